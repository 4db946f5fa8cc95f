"""Korurax on the host side, without a GPU: its configuration (every key read, faults named), its weights, the model as
data (what each layer keeps), pages that a chunk has passed, and the whole path through cache manager, step function and
replay on the CPU with the kernels replaced by their PyTorch statements."""
import copy
import io
import json

import numpy as np
import pytest
import torch

import plain_korurax as plain
import replay_cases as rc


@pytest.fixture(scope="module")
def model_a(tmp_path_factory):
  return plain.make_model_dir(plain.CONFIGS["A"], str(tmp_path_factory.mktemp("korurax_A")), seed=3)


def test_configuration_is_read_key_by_key(model_a):
  from miniinfer_b200.config import KoruraxConfig, load_model_config
  cfg = load_model_config(model_a)
  assert isinstance(cfg, KoruraxConfig)
  assert (cfg.vocab_size, cfg.width, cfg.norm_eps, cfg.residual_mult, cfg.logit_softcap) == (300, 64, 1e-5, 0.5, 20.0)
  a, l = cfg.mixer_of(0), cfg.mixer_of(1)
  assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk) == (4, 1, 24, 40, 0.3, 24)
  assert (l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.scale, l.rot.dims, l.rot.base) == (3, 24, 8, 16, 24, 40, 0.2, 8, 10000.0)
  d, m = cfg.mlp_of(0), cfg.mlp_of(1)
  assert (d.kind, d.ff, d.limit) == ("dense", 40, 1.5) and (m.kind, m.ff, m.experts, m.top, m.scale) == ("moe", 24, 5, 2, 2.5)
  assert cfg.mlp_of(2) is None and cfg.to_dict() == plain.CONFIGS["A"]


@pytest.mark.parametrize("change,key", [
  (lambda c: c["layers"][0].__setitem__("type", "gla"), "layers[0].type"),
  (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "mixer.heads"),
  (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "mask.size"),
  (lambda c: c["layers"][0]["mixer"].__setitem__("mask", 24), "mixer.mask"),
  (lambda c: c["layers"][0]["mixer"].pop("scale"), "mixer.scale"),
  (lambda c: c["layers"][0]["mlp"].pop("limit"), "mlp.limit"),
  (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "wide"), "mlp.kind"),
  (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 4), "rot.dims"),
  (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "mixer.q_rank"),
  (lambda c: c["layers"][1]["mixer"].pop("rot"), "mixer.rot"),
  (lambda c: c["layers"][1]["mlp"]["router"].__setitem__("top", 9), "router.top"),
  (lambda c: c["layers"][1]["mlp"]["router"].pop("scale"), "router.scale"),
  (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
  (lambda c: c.__setitem__("residual_mult", None), "residual_mult"),
  (lambda c: c.__setitem__("logit_softcap", 0), "logit_softcap"),
  (lambda c: c.pop("logit_softcap"), "logit_softcap"),
  (lambda c: c["norm"].__setitem__("eps", 0), "norm.eps"),
  (lambda c: c.__setitem__("width", 0), "width"),
  (lambda c: c.__setitem__("layers", []), "layers"),
])
def test_faulty_configurations_are_refused_with_the_key(change, key):
  from miniinfer_b200.config import ConfigError, KoruraxConfig
  c = copy.deepcopy(plain.CONFIGS["A"])
  change(c)
  with pytest.raises(ConfigError) as e:
    KoruraxConfig.from_dict(c)
  assert key in str(e.value)


def test_the_model_as_data(model_a):
  from miniinfer_b200.cache.specs import PagedKVSpec
  from miniinfer_b200.config import build_model_spec, load_model_config
  from miniinfer_b200.parts import (DepthAverageBlock, DepthAverageNorm, GatedAttentionMixer, LatentAttentionMixer, RoutedExpertsFeedForward,
                                    SwiGLUFeedForward)
  spec = build_model_spec(load_model_config(model_a))
  assert [type(b.mixer) for b in spec.blocks] == [GatedAttentionMixer, LatentAttentionMixer, GatedAttentionMixer, LatentAttentionMixer, GatedAttentionMixer]
  assert all(isinstance(b, DepthAverageBlock) and (b.index, b.depth, b.mult) == (i, 5, 0.5) for i, b in enumerate(spec.blocks))
  att, lat = spec.blocks[0].mixer, spec.blocks[1].mixer
  assert att.sinks and att.gated and att.gate_per_head and att.distance_bias and att.chunk == 24 and att.qk_norm_eps is None and att.position is None
  assert att.proj_width % 8 == 0 and att.proj_width - (4 * 24 + 24 + 40 + 4) < 8
  assert not lat.sinks and not lat.gated and lat.down_width == 24 + 40 + 8
  # rows of max(dim, vdim) padded to 16; a latent's of kv_rank + rot_dim
  assert spec.cache_layer_specs() == [PagedKVSpec(1, 48, chunk=24), PagedKVSpec(1, 48), PagedKVSpec(1, 48, chunk=24), PagedKVSpec(1, 48), PagedKVSpec(2, 16, chunk=50)]
  assert spec.blocks[1].mixer.position is spec.blocks[3].mixer.position and len(spec.position_encodings) == 1
  d, m = spec.blocks[0].ffn, spec.blocks[1].ffn
  assert isinstance(d, SwiGLUFeedForward) and (d.activation, d.limit) == ("clamped", 1.5) and spec.blocks[2].ffn is None
  assert isinstance(m, RoutedExpertsFeedForward) and (m.activation, m.has_correction, m.weight_scale, m.gated) == ("relu_squared", False, 2.5, False)
  assert isinstance(spec.final_norm, DepthAverageNorm) and spec.lm_head.tied_to is spec.embedding and spec.lm_head.softcap == 20.0
  assert spec.unused == ["l2.norm2"]


def test_weights_are_asked_for_by_name(model_a, tmp_path):
  from safetensors.torch import load_file, save_file
  from miniinfer_b200.config import build_model_spec, load_model_config
  from miniinfer_b200.weights import WeightLoadError, load_weights
  spec = build_model_spec(load_model_config(model_a))
  load_weights(spec, model_a, torch.float32, "cpu")
  W = plain.read_weights(model_a)
  a = spec.blocks[4].mixer                    # two heads of 16, two key/value heads: 96 columns and two gates, padded to 104
  assert a.qkvg.shape == (104, 64) and torch.equal(a.qkvg[96:98], W["l4.mix.g"]) and not a.qkvg[98:].any()
  assert torch.equal(a.distance, torch.cat([W["l4.mix.r1"], W["l4.mix.r2"]])) and torch.equal(a.sink, W["l4.mix.sink"])
  assert torch.equal(spec.blocks[3].weights, W["l3.dwa"]) and torch.equal(spec.blocks[1].ffn.gate_up[24:48], W["l1.mlp.e1.up"])
  assert torch.equal(spec.final_norm.norm.weight, W["final.norm"]) and spec.final_norm.norm.bias is None
  raw = load_file(f"{model_a}/model.safetensors")
  raw.pop("l0.mix.r2")
  raw["l2.norm2"] = raw["l2.norm1"].clone()                   # a norm in front of a feed-forward that is not there may be present
  raw["l1.mlp.correction"] = torch.zeros(5)
  raw["l3.dwa"] = raw["l3.dwa"][:4].contiguous()
  d = tmp_path / "broken"
  d.mkdir()
  (d / "config.json").write_text(json.dumps(plain.CONFIGS["A"]))
  save_file(raw, str(d / "model.safetensors"))
  with pytest.raises(WeightLoadError) as e:
    load_weights(build_model_spec(load_model_config(str(d))), str(d), torch.bfloat16, "cpu")
  assert e.value.missing == ["l0.mix.r2"] and e.value.unexpected == ["l1.mlp.correction"] and "l3.dwa" in e.value.wrong_shape[0]


def test_random_weights_mode_writes_a_model_of_the_design(tmp_path):
  from miniinfer_b200.weights import write_random_model
  d = write_random_model(copy.deepcopy(plain.CONFIGS["B"]), str(tmp_path / "m"), seed=4)
  W, cfg = plain.read_weights(d), plain.read_config(d)
  assert set(W) == set(plain.tensor_shapes(plain.CONFIGS["B"])) and all(tuple(W[k].shape) == s for k, s in plain.tensor_shapes(plain.CONFIGS["B"]).items())
  assert torch.isfinite(plain.forward(cfg, W, [1, 2, 3])).all()


def test_pages_that_a_chunk_has_passed_go_back():
  from miniinfer_b200.cache.manager import KVCacheManager
  from miniinfer_b200.cache.specs import PagedKVSpec
  m = KVCacheManager([PagedKVSpec(1, 16), PagedKVSpec(1, 16, chunk=24)], 16, 20, 2, 320, torch.float32)
  m.admit("a")
  held = lambda: [i for i, p in enumerate(m._requests["a"].pages[1]) if p]
  for n, pages in ((23, [0, 1]), (1, [1]), (7, [1]), (1, [1]), (15, [1, 2]), (1, []), (1, [3]), (31, [4])):
    # the next query, at position `length`, sees its chunk of 24 positions from floor(length / 24) * 24 on
    m.append("a", n)
    m.commit("a", n)
    assert held() == pages, (m.length_of("a"), held())
    m.check_invariants()
  assert len([p for p in m._requests["a"].pages[0] if p]) == 5      # the group that keeps every key gives nothing back
  m.release_request("a")
  assert m.free_pages() == [20, 20]
  assert KVCacheManager.group_pages(PagedKVSpec(1, 16, chunk=32), 16, 1000, 4, 64) == 4 * 11      # a chunk and what two steps of 64 tokens add
  for bad in (dict(chunk=0), dict(chunk=8, window=8)):
    with pytest.raises(ValueError):
      PagedKVSpec(1, 16, **bad)


def test_parts_refuse_options_that_do_not_go_together():
  from miniinfer_b200.parts import DepthAverageBlock, GatedAttentionMixer, LMHead, RoutedExpertsFeedForward, SwiGLUFeedForward
  with pytest.raises(ValueError, match="chunk"):
    GatedAttentionMixer("m", 32, 2, 1, 16, 16, 1.0, None, window=8, chunk=8)
  with pytest.raises(ValueError, match="distance"):
    GatedAttentionMixer("m", 32, 2, 1, 16, 16, 1.0, None, sinks=False, weights="sigmoid", distance_bias=True)
  with pytest.raises(ValueError, match="gate_per_head"):
    GatedAttentionMixer("m", 32, 2, 1, 16, 16, 1.0, None, gated=False, gate_per_head=True)
  with pytest.raises(ValueError, match="limit"):
    SwiGLUFeedForward("f", 32, 16, activation="clamped")
  with pytest.raises(ValueError, match="shared"):
    RoutedExpertsFeedForward("f", 32, 16, 4, 2, activation="relu_squared", shared_size=8)
  with pytest.raises(ValueError, match="index"):
    DepthAverageBlock("b", 3, 3, 32, None, None, None, None)
  with pytest.raises(ValueError, match="softcap"):
    LMHead("h", 10, 32, softcap=-1.0)


def _mistakes():
  """(what, change of configuration and weights) of mistakes in single mechanisms, planted in the plain implementation."""
  def chunk(d):
    return lambda c, W: [x["mixer"]["mask"].__setitem__("size", x["mixer"]["mask"]["size"] + d) for x in c["layers"] if x["type"] == "attention"]

  def scale(suffix, f):
    return lambda c, W: W.update({k: f(v) for k, v in W.items() if k.endswith(suffix)})

  return [("chunks one longer", chunk(1)), ("chunks one shorter", chunk(-1)), ("no chunks", chunk(100000)),
          ("no sink", scale(".sink", lambda v: v - 100.0)), ("no distance bias", scale(".r1", lambda v: v * 0)),
          ("distances half", scale(".r2", lambda v: v * 0.5)), ("gates open", scale("mix.g", lambda v: v * 0)),
          ("no rotation", lambda c, W: [x["mixer"]["rot"].__setitem__("base", 1e30) for x in c["layers"] if "rot" in x["mixer"]]),
          ("the last layer alone", scale(".dwa", lambda v: torch.cat((v[:-1] * 0, v[-1:])))),
          ("no multiplier", lambda c, W: c.__setitem__("residual_mult", 1.0)), ("no cap", lambda c, W: c.__setitem__("logit_softcap", 1e6)),
          ("another limit", lambda c, W: [x["mlp"].__setitem__("limit", 1e6) for x in c["layers"] if x["mlp"] and x["mlp"]["kind"] == "dense"]),
          ("another share", lambda c, W: [x["mlp"]["router"].__setitem__("scale", 1.25) for x in c["layers"] if x["mlp"] and x["mlp"]["kind"] == "moe"])]


@pytest.mark.parametrize("k", range(13))
def test_a_mistake_in_one_mechanism_would_show(k):
  """The weights that the GPU tests run on let every mechanism show: the plain logits with a mistake planted in one of them
  differ from those without by many times the bound that the engine's float32 logits are held to."""
  what, change = _mistakes()[k]
  cfg, W = plain.peaky_model()
  ids = torch.randint(0, cfg["vocab"], (310,), generator=torch.Generator().manual_seed(6)).tolist()
  ref = plain.forward(cfg, W, ids)
  c2, W2 = copy.deepcopy(cfg), dict(W)
  change(c2, W2)
  diff = (plain.forward(c2, W2, ids) - ref).abs().max(-1).values
  bound = 3e-4 * max(1.0, float(ref.pow(2).mean().sqrt()))
  first = {"chunks one longer": 100, "chunks one shorter": 99, "no chunks": 100}.get(what)
  if first is not None:      # an edge that is one off moves nothing before it, and the tokens behind it
    assert float(diff[:69].max()) == 0
  assert float((diff > 20 * bound).float().mean()) > (0.02 if first else 0.3), (what, float(diff.max()), bound)


@pytest.mark.parametrize("tag,page", [("A", 16), ("B", 8), ("C", 64), ("D", 16), ("E", 64)])
def test_every_cut_gives_the_plain_logits_on_the_host_path(cpu_kernels, tmp_path, tag, page):
  from miniinfer_b200.engine.replay import TraceRunner
  cfg = plain.CONFIGS[tag]
  d = plain.make_model_dir(cfg, str(tmp_path / tag), seed=8)
  lengths = (5, 17, 33, 70, 64, 41, 2, 1)
  reqs = rc.make_requests(cfg["vocab"], lengths, seed=5)
  W = plain.read_weights(d)
  ref = {rid: plain.forward(cfg, W, ids) for rid, ids in reqs.items()}
  budget = 2 * rc.round_up(max(lengths), page)
  for name, trace in (("whole", rc.whole(reqs)), ("tail", rc.tail_one_by_one(reqs)), ("portions", rc.portions(reqs)),
                      ("mixed", rc.mixed(reqs, budget, seed=1, granule=page)),
                      ("preempted", rc.mixed(reqs, budget, seed=2, granule=page, preempt=True))):
    runner = TraceRunner(d, "float32", budget, device="cpu", page_size=page, max_requests=4)
    got = rc.run_in_process(runner, trace)
    rc.compare(got, ref, 2e-3, f"korurax {tag}/{name}")
    runner.cache.check_invariants()
    assert runner.cache.free_pages() == [g.num_pages for g in runner.cache.paged_groups]


def test_trace_program_picks_the_model_by_its_configuration(cpu_kernels, model_a, tmp_path):
  from miniinfer_b200.engine import replay
  reqs = rc.make_requests(300, (20, 9), seed=2)
  trace = rc.mixed(reqs, 128, seed=3)
  out = io.StringIO()
  code = replay.main(["--model", model_a, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "128",
                      "--device", "cpu"], stdin=io.StringIO("\n".join(json.dumps(r) for r in trace) + "\n"), stdout=out)
  assert code == 0 and out.getvalue().split("\n")[:-1] == [f"done {r['step']}" for r in trace]
  outputs = {r["step"]: np.fromfile(tmp_path / "o" / f"{r['step']}.f32", dtype="<f4").reshape(-1, 300)
             for r in trace if sum(len(e["want"]) for e in r["entries"])}
  W, cfg = plain.read_weights(model_a), plain.read_config(model_a)
  rc.compare(rc.collect(trace, outputs), {rid: plain.forward(cfg, W, ids) for rid, ids in reqs.items()}, 2e-3, "trace program")
