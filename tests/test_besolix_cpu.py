"""Besolix on the host side, without a GPU: its configuration (every key read, faults named), its weights, the model as
data (what each layer keeps, and who reads whose), and the whole path through cache manager, step function and replay on
the CPU with the kernels replaced by their PyTorch statements."""
import copy
import io
import json

import numpy as np
import pytest
import torch

import plain_besolix as plain
import replay_cases as rc


@pytest.fixture(scope="module")
def model_a(tmp_path_factory):
  return plain.make_model_dir(plain.CONFIGS["A"], str(tmp_path_factory.mktemp("besolix_A")), seed=3)


def test_configuration_is_read_key_by_key(model_a):
  from miniinfer_b200.config import BesolixConfig, load_model_config
  cfg = load_model_config(model_a)
  assert isinstance(cfg, BesolixConfig) and (cfg.vocab_size, cfg.width, cfg.norm_eps) == (300, 64, 1e-5)
  l, a, d, r = (cfg.mixer_of(i) for i in range(4))
  assert (l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.scale, l.window, l.kv_from) == (3, 24, 8, 16, 24, 40, 0.2, 24, None)
  assert (l.rot.dims, l.rot.base, l.rot.scaling) == (8, 10000.0, None)
  assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window) == (4, 1, 24, 40, 0.25, 20)
  assert (a.rot.dims, a.rot.base, a.rot.scaling) == (16, 5000.0, {"factor": 4.0})
  assert (d.heads, d.kv_heads, d.dim, d.vdim, d.conv) == (4, 2, 16, 24, 4)
  assert (r.heads, r.window, r.kv_from) == (5, 50, 0)
  assert [cfg.ff_of(i) for i in range(6)] == [40, 48, 40, None, None, 24] and cfg.to_dict() == plain.CONFIGS["A"]


@pytest.mark.parametrize("change,key", [
  (lambda c: c["layers"][0].__setitem__("type", "gla"), "layers[0].type"),
  (lambda c: c["layers"][1]["mixer"].__setitem__("kv_heads", 3), "mixer.heads"),
  (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", 0), "mask.size"),
  (lambda c: c["layers"][1]["mixer"].__setitem__("mask", 24), "mixer.mask"),
  (lambda c: c["layers"][1]["mixer"].pop("scale"), "mixer.scale"),
  (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 26), "rot.dims"),
  (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 5), "rot.dims"),
  (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("factor"), "scaling.factor"),
  (lambda c: c["layers"][1]["mixer"].pop("rot"), "mixer.rot"),
  (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 4), "rot.dims"),
  (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "mixer.q_rank"),
  (lambda c: c["layers"][2]["mixer"].pop("conv"), "mixer.conv"),
  (lambda c: c["layers"][2]["mixer"].__setitem__("kv_heads", 3), "mixer.heads"),
  (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 3), "kv_from"),
  (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 1), "kv_from"),
  (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", -1), "kv_from"),
  (lambda c: c["layers"][3]["mixer"].__setitem__("kv_rank", 48), "kv_rank"),
  (lambda c: c["layers"][3]["mixer"]["rot"].__setitem__("base", 5.0), "rot"),
  (lambda c: c["layers"].append(plain.latent(3, 24, 8, 16, 24, 40, 24, 10000.0, 0.2, None, kv_from=3)), "kv_from"),
  (lambda c: c["layers"][0]["mlp"].pop("ff"), "mlp.ff"),
  (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "mlp.kind"),
  (lambda c: c["norm"].__setitem__("eps", 0), "norm.eps"),
  (lambda c: c.__setitem__("width", 0), "width"),
  (lambda c: c.__setitem__("layers", []), "layers"),
])
def test_faulty_configurations_are_refused_with_the_key(change, key):
  from miniinfer_b200.config import BesolixConfig, ConfigError
  c = copy.deepcopy(plain.CONFIGS["A"])
  change(c)
  with pytest.raises(ConfigError) as e:
    BesolixConfig.from_dict(c)
  assert key in str(e.value)


def test_the_model_as_data(model_a):
  from miniinfer_b200.cache.specs import FixedStateSpec, PagedKVSpec
  from miniinfer_b200.config import build_model_spec, load_model_config
  from miniinfer_b200.parts import GatedAttentionMixer, GatedDeltaMixer, LatentAttentionMixer, PreNormBlock, SwiGLUFeedForward
  spec = build_model_spec(load_model_config(model_a))
  assert [type(b.mixer) for b in spec.blocks] == [LatentAttentionMixer, GatedAttentionMixer, GatedDeltaMixer, LatentAttentionMixer, GatedDeltaMixer,
                                                  GatedAttentionMixer]
  assert all(isinstance(b, PreNormBlock) and b.mixer_norm.offset == 1.0 for b in spec.blocks)
  lat, att, dlt, rdr = (spec.blocks[i].mixer for i in range(4))
  assert not lat.sinks and lat.gated and not lat.gate_per_head and lat.keeps_latents and lat.rotary_interleaved
  assert lat.down_width == 24 + 40 + 8 + 3 * 16 and rdr.down_width == 32 + 5 * 24 and not rdr.keeps_latents
  assert "dkv_norm" in lat.param_specs() and "dkv_norm" not in rdr.param_specs()
  assert att.norm_weights and att.rotary_interleaved and not att.sinks and not att.gated and att.window == 20
  assert dlt.decay_rank is None and dlt.gate_rank is None and dlt.gate_silu and dlt.proj_width % 8 == 0
  # the cache of layer 0 is kept for the window of its reader, which is the wider one
  state = FixedStateSpec((3 * (2 * 2 * 16 + 4 * 24) + 4 * 16 * 24,))
  assert spec.cache_layer_specs() == [PagedKVSpec(1, 48, 50), PagedKVSpec(1, 48, 20), state, None, state, PagedKVSpec(1, 48, 20)]
  assert [(r.block, r.cache_of) for r in spec.run_list] == [(0, None), (1, None), (2, None), (3, 0), (4, None), (5, None)]
  assert lat.position is rdr.position and len(spec.position_encodings) == 2
  f = spec.blocks[0].ffn
  assert isinstance(f, SwiGLUFeedForward) and f.activation == "gelu_tanh" and spec.blocks[3].ffn is None
  assert spec.lm_head.tied_to is None and spec.unused == ["l3.norm2", "l4.norm2"]


def test_a_cache_is_kept_for_the_widest_of_its_readers():
  from miniinfer_b200.cache.specs import FixedStateSpec, PagedKVSpec, shared_need
  from miniinfer_b200.config import BesolixConfig, build_model_spec
  P = PagedKVSpec
  assert shared_need([P(1, 48, 9), P(1, 48, 9)]) == P(1, 48, 9)
  assert shared_need([P(1, 48, 9), P(1, 48, 30), P(1, 48, 12, 5)]) == P(1, 48, 30, 5)
  assert shared_need([P(1, 48, 9), P(1, 48)]) == P(1, 48) and shared_need([P(1, 48, 9), P(1, 48, chunk=9)]) == P(1, 48)
  assert shared_need([P(1, 48, chunk=9), P(1, 48, chunk=9)]) == P(1, 48, chunk=9) and shared_need([P(1, 48, chunk=9), P(1, 48, chunk=8)]) == P(1, 48)
  for bad in ([P(1, 48), P(2, 48)], [P(1, 48), P(1, 64)], [P(1, 48), FixedStateSpec((3,))]):
    with pytest.raises(ValueError):
      shared_need(bad)
  keeps = lambda tag: build_model_spec(BesolixConfig.from_dict(copy.deepcopy(plain.CONFIGS[tag]))).cache_layer_specs()
  assert keeps("B")[1] == P(1, 32) and keeps("B")[3] is None and keeps("B")[5] is None      # one reader sees every earlier token
  assert keeps("E")[:3] == [P(1, 128, 200), None, None]
  assert keeps("D")[0] == P(1, 272, 40) and keeps("D")[1] == P(1, 48, 17)


def test_weights_are_asked_for_by_name(model_a, tmp_path):
  from safetensors.torch import load_file, save_file
  from miniinfer_b200.config import build_model_spec, load_model_config
  from miniinfer_b200.weights import WeightLoadError, load_weights
  spec = build_model_spec(load_model_config(model_a))
  load_weights(spec, model_a, torch.float32, "cpu")
  W = plain.read_weights(model_a)
  lat, dlt, rdr = (spec.blocks[i].mixer for i in (0, 2, 3))
  assert torch.equal(lat.down[24:72], W["l0.mix.dkv"]) and torch.equal(lat.down[72:], W["l0.mix.g"]) and torch.equal(rdr.down[32:], W["l3.mix.g"])
  assert torch.equal(dlt.proj[:96], W["l2.mix.g"]) and torch.equal(dlt.proj[96:128], W["l2.mix.q"]) and torch.equal(dlt.proj[256:260], W["l2.mix.b"])
  assert torch.equal(dlt.proj[260:264], W["l2.mix.a"]) and torch.equal(dlt.conv[64:], W["l2.mix.v.conv"]) and dlt.dt_bias.shape == (4,)
  assert torch.equal(spec.final_norm.weight, 1.0 + W["final.norm"]) and torch.equal(spec.lm_head.weight, W["head"])
  raw = load_file(f"{model_a}/model.safetensors")
  raw.pop("l2.mix.a")
  raw["l3.norm2"] = raw["l3.norm1"].clone()                   # a norm in front of a feed-forward that is not there may be present
  raw["l3.mix.dkv"] = raw["l0.mix.dkv"].clone()               # a reader has no latents of its own
  raw["l2.mix.dt_bias"] = torch.zeros(64, dtype=torch.bfloat16)
  d = tmp_path / "broken"
  d.mkdir()
  (d / "config.json").write_text(json.dumps(plain.CONFIGS["A"]))
  save_file(raw, str(d / "model.safetensors"))
  with pytest.raises(WeightLoadError) as e:
    load_weights(build_model_spec(load_model_config(str(d))), str(d), torch.bfloat16, "cpu")
  assert e.value.missing == ["l2.mix.a"] and e.value.unexpected == ["l3.mix.dkv"] and "l2.mix.dt_bias" in e.value.wrong_shape[0]


def test_random_weights_mode_writes_a_model_of_the_design(tmp_path):
  from miniinfer_b200.weights import write_random_model
  d = write_random_model(copy.deepcopy(plain.CONFIGS["B"]), str(tmp_path / "m"), seed=4)
  W, cfg = plain.read_weights(d), plain.read_config(d)
  assert set(W) == set(plain.tensor_shapes(plain.CONFIGS["B"])) and all(tuple(W[k].shape) == s for k, s in plain.tensor_shapes(plain.CONFIGS["B"]).items())
  assert torch.isfinite(plain.forward(cfg, W, [1, 2, 3])).all()


def test_divided_rotary_frequencies():
  from miniinfer_b200.parts import LinearScaledRotaryEncoding
  for dims, base, factor in ((16, 5000.0, 4.0), (24, 50.0, 1.0), (2, 300.0, 2.5)):
    table = LinearScaledRotaryEncoding("rot", dims, base, 4096, factor=factor).build_table(300)
    x = torch.randn((300, 1, dims), generator=torch.Generator().manual_seed(dims), dtype=torch.float64)
    want = plain.rotate_pairs(x, torch.arange(300), dims, base, factor)[:, 0]
    c, s = table[:, :dims // 2].double(), table[:, dims // 2:].double()
    u, v = x[:, 0, 0::2], x[:, 0, 1::2]
    assert float((torch.stack([u * c - v * s, v * c + u * s], -1).flatten(1) - want).abs().max()) < 1e-6
  with pytest.raises(ValueError, match="factor"):
    LinearScaledRotaryEncoding("rot", 8, 100.0, 64, factor=0.0)


def test_parts_refuse_options_that_do_not_go_together():
  from miniinfer_b200.parts import GatedDeltaMixer, LatentAttentionMixer, LinearScaledRotaryEncoding, SwiGLUFeedForward
  from miniinfer_b200.cache.manager import LayerCache
  with pytest.raises(ValueError, match="gate"):
    GatedDeltaMixer("m", 32, 2, 1, 16, 16, 2, None, None, 1e-6, gate="relu")
  with pytest.raises(ValueError, match="decay_rank"):
    GatedDeltaMixer("m", 32, 2, 1, 16, 16, 2, 0, None, 1e-6)
  with pytest.raises(ValueError, match="activation"):
    SwiGLUFeedForward("f", 32, 16, activation="gelu")
  reader = LatentAttentionMixer("m", 32, 2, 16, 8, 16, 8, 16, 1.0, 1e-6, LinearScaledRotaryEncoding("r", 8, 100.0, 64), keeps_latents=False)
  with pytest.raises(RuntimeError, match="another layer"):
    reader.forward(torch.zeros(1, 32), None, LayerCache("paged", 0, None, True, 16))


def test_a_run_list_entry_cannot_read_rows_of_another_shape():
  from miniinfer_b200.config import BesolixConfig, build_model_spec
  from miniinfer_b200.models import LayerRun, ModelSpec
  spec = build_model_spec(BesolixConfig.from_dict(copy.deepcopy(plain.CONFIGS["B"])))
  args = dict(config=spec.config, embedding=spec.embedding, blocks=spec.blocks, final_norm=spec.final_norm, lm_head=spec.lm_head)
  with pytest.raises(ValueError, match="keep in the cache"):
    ModelSpec(**args, run_list=[LayerRun(1), LayerRun(4, cache_of=0)])
  with pytest.raises(ValueError, match="none of its own"):
    ModelSpec(**args, run_list=[LayerRun(1), LayerRun(3, cache_of=0), LayerRun(5, cache_of=1)])


def _mistakes():
  """(what, change of configuration and weights) of mistakes in single mechanisms, planted in the plain implementation."""
  def window(kind, d):
    return lambda c, W: [x["mixer"]["mask"].__setitem__("size", x["mixer"]["mask"]["size"] + d) for x in c["layers"] if x["type"] == kind]

  def each(suffix, f):
    return lambda c, W: W.update({k: f(v) for k, v in W.items() if k.endswith(suffix)})

  def mixers(key, v):
    return lambda c, W: [x["mixer"].__setitem__(key, v) for x in c["layers"] if key in x["mixer"]]

  def own_latents(c, W):
    c["layers"][2]["mixer"].pop("kv_from")
    W.update({"l2.mix.dkv": W["l0.mix.dkv"], "l2.mix.dkv.norm": W["l0.mix.dkv.norm"]})

  def scale_conv(v):
    return torch.cat([v[:, :-1] * 0, v[:, -1:]], 1)

  return [("latent windows one longer", window("latent_attention", 1)), ("latent windows one shorter", window("latent_attention", -1)),
          ("windows one longer", window("attention", 1)), ("windows one shorter", window("attention", -1)),
          ("latents made anew from the later layer's input", own_latents),
          ("latent gates half open", each("l0.mix.g", lambda v: v * 0)), ("delta gates shut", each("l3.mix.g", lambda v: v * 0)),
          ("no rotation", lambda c, W: [x["mixer"]["rot"].__setitem__("base", 1e30) for x in c["layers"] if "rot" in x["mixer"]]),
          ("frequencies not divided", lambda c, W: c["layers"][1]["mixer"]["rot"].pop("scaling")),
          ("one rotated pair fewer", lambda c, W: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 22)),
          ("no decay", each("A_log", lambda v: v - 50.0)), ("decays without their bias", each("dt_bias", lambda v: v * 0)),
          ("half as much written", each("mix.b", lambda v: v * 0)), ("convolutions of the last tap alone", each(".conv", scale_conv)),
          ("norms as stored", lambda c, W: W.update({k: v - 1.0 for k, v in W.items() if k.split(".")[-1] in ("norm1", "norm2") or k == "final.norm"})),
          ("query norms without a weight", each("q.norm", lambda v: v * 0 + 1.0)), ("another scale", mixers("scale", 0.4))]


@pytest.mark.parametrize("k", range(17))
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
  edge = "window" in what
  if edge:      # an edge that is one off moves nothing before it, and the tokens behind it
    assert float(diff[:69].max()) == 0
  assert float((diff > 20 * bound).float().mean()) > (0.02 if edge else 0.3), (what, float(diff.max()), bound)


@pytest.mark.parametrize("tag,page", [("A", 16), ("B", 8), ("C", 64), ("D", 16), ("E", 64), ("F", 8)])
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
    rc.compare(got, ref, 2e-3, f"besolix {tag}/{name}")
    runner.cache.check_invariants()
    assert runner.cache.free_pages() == [g.num_pages for g in runner.cache.paged_groups]


def test_pages_stay_until_the_last_reader_has_passed_them(cpu_kernels, model_a):
  """Layer 0 looks back 24 tokens, its reader 50: a page of layer 0's group goes back when both have passed it."""
  from miniinfer_b200.engine.replay import TraceRunner
  runner = TraceRunner(model_a, "float32", 128, device="cpu", page_size=16, max_requests=2)
  ids = torch.randint(0, 300, (100,), generator=torch.Generator().manual_seed(1)).tolist()
  group = next(g for g in runner.cache.paged_groups if g.spec.window == 50)
  other = next(g for g in runner.cache.paged_groups if g.spec.window == 20)
  for n, (lo, hi) in enumerate(((0, 65), (65, 66), (66, 100))):
    runner.run_step({"entries": [{"id": "a", "tokens": ids[lo:hi], "want": []}]})
    first = [next(i for i, p in enumerate(runner.cache._requests["a"].pages[g.index]) if p) for g in (group, other)]
    assert first == [max(0, hi - 49) // 16, max(0, hi - 19) // 16]
  runner.cache.check_invariants()


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
