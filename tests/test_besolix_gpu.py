"""The Besolix design in the engine against its plain implementation (tests/plain_besolix.py): every way of cutting
requests into steps, in float32 and bfloat16, on configurations that differ in every size, in the order of their layers
and in who reads whose latents; long decoding over many windows with their pages given back and handed out again while
other layers still read theirs; single keys that stand out far back, at page borders and on both sides of every window's
edge; recurrent state over pauses, portions and slots that are used again; greedy generation through the entry point and
its scheduler."""
import copy

import numpy as np
import pytest
import torch

import plain_besolix as plain
import replay_cases as rc
from gpu_helpers import DEV

pytestmark = pytest.mark.gpu

LENGTHS = {"A": (5, 17, 33, 100, 64, 128, 41, 65, 1, 2), "B": (1, 9, 40, 71, 130, 65, 200, 2), "C": (130, 70, 300, 64, 200, 65, 257, 1),
           "D": (3, 50, 129, 70, 1, 16), "E": (300, 131, 201, 64, 1, 270), "F": (1, 30, 90, 17, 2, 65)}
PAGES = {"A": 16, "B": 16, "C": 64, "D": 16, "E": 64, "F": 8}
# bfloat16, as fractions of the root mean square of the plain logits: rounding every product to bfloat16 moves a row by a
# few hundredths of that, and a first token, whose short row the delta rule's unit norms blow up, by more; a wrong key, a
# window's edge one off or a lost state moves most rows by tenths, and shows in the float32 runs, which take the same path
# through the engine and allow nothing.
BF16_MEDIAN, BF16_BOUND, BF16_CAP = 0.03, 0.12, 1.0


@pytest.fixture(scope="module")
def besolix_dirs(tmp_path_factory):
  made = {}

  def get(tag):
    if tag not in made:
      made[tag] = plain.make_model_dir(plain.CONFIGS[tag], str(tmp_path_factory.mktemp(f"besolix_{tag}")), seed=71 + len(made))
    return made[tag]

  return get


_refs = {}


def reference(model_dir, reqs):
  key = (model_dir, tuple(sorted(reqs)), tuple(len(v) for v in reqs.values()))
  if key not in _refs:
    W, cfg = plain.read_weights(model_dir), plain.read_config(model_dir)
    with torch.no_grad():
      _refs[key] = {rid: plain.forward(cfg, W, ids) for rid, ids in reqs.items()}
  return _refs[key]


def runner_for(model_dir, dtype, max_tokens, page, max_requests=4):
  from miniinfer_b200.engine.replay import TraceRunner
  return TraceRunner(model_dir, dtype, max_tokens, device=DEV, page_size=page, max_requests=max_requests)


def compare(got, ref, dtype, what):
  size = float(np.sqrt(np.mean([float(r.pow(2).mean()) for r in ref.values()])))
  if dtype == "float32":
    rc.compare(got, ref, 3e-4 * max(1.0, size), what, check_argmax_margin=2e-3 * max(1.0, size))
    return
  assert got, "nothing was compared"
  errs = []
  for key, row in sorted(got.items()):
    assert np.isfinite(row).all(), f"{what}: request {key[0]} position {key[1]}: logits are not finite"
    d = row - ref[key[0]][key[1]].numpy()
    errs.append(float(np.sqrt(((d - d.mean()) ** 2).mean())) / size)       # root mean square of the centred difference
    assert errs[-1] <= BF16_CAP, f"{what}: request {key[0]} position {key[1]}: the row differs by {errs[-1]:.3f}"
  errs = np.array(errs)
  assert np.median(errs) <= BF16_MEDIAN, f"{what}: the middle row differs by {np.median(errs):.4f}"
  assert (errs > BF16_BOUND).sum() <= max(2, 0.08 * len(errs)), f"{what}: {(errs > BF16_BOUND).sum()} of {len(errs)} rows differ by more than {BF16_BOUND}"
  rc.log_worst(what, float(errs.max()), ref)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "B", "C", "D", "E", "F"])
@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "mixed", "preempted"])
def test_every_cut_gives_the_plain_logits(besolix_dirs, dtype, tag, cut):
  d = besolix_dirs(tag)
  page = PAGES[tag]
  reqs = rc.make_requests(plain.CONFIGS[tag]["vocab"], LENGTHS[tag], seed=5)
  ref = reference(d, reqs)
  longest = rc.round_up(max(LENGTHS[tag]), page)
  if cut in ("mixed", "preempted"):
    budget = longest + 2 * rc.round_up(70, page)      # requests wait for pages that others give back
    trace = rc.mixed(reqs, budget, seed=1, granule=page, preempt=cut == "preempted")
    assert max(len(r["entries"]) for r in trace) >= 2
  else:
    budget = longest
    trace = {"whole": rc.whole, "tail": rc.tail_one_by_one, "portions": rc.portions}[cut](reqs)
  runner = runner_for(d, dtype, budget, page)
  got = rc.run_in_process(runner, trace)
  compare(got, ref, dtype, f"besolix {tag}/{dtype}/{cut}")
  runner.cache.check_invariants()
  assert runner.cache.free_pages() == [g.num_pages for g in runner.cache.paged_groups]
  runner.runner.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "B"])
def test_long_decoding_over_page_borders(besolix_dirs, dtype, tag):
  """Twelve tokens as a prompt, then 250 tokens one by one over many windows and page borders (pages of 8): pages that a
  window has passed go back and are handed out again while layers with wider windows still read theirs, and the recurrent
  state and the convolutions' last inputs go on from token to token; a second request - portions of three tokens, then single
  ones - runs beside the first from step 100 on."""
  d = besolix_dirs(tag)
  reqs = rc.make_requests(plain.CONFIGS[tag]["vocab"], (262, 150), seed=9)
  ref = reference(d, reqs)
  a, b = reqs["r0"], reqs["r1"]
  trace = [{"step": 0, "entries": [{"id": "r0", "tokens": a[:12], "want": list(range(12))}], "end": []}]
  pos_b = 0
  for j in range(12, len(a)):
    entries = [{"id": "r0", "tokens": [a[j]], "want": [0]}]
    if j >= 100 and pos_b < len(b):
      n = 3 if pos_b < 30 else 1
      entries.append({"id": "r1", "tokens": b[pos_b:pos_b + n], "want": list(range(len(b[pos_b:pos_b + n])))})
      pos_b += n
    trace.append({"step": len(trace), "entries": entries, "end": []})
  trace[-1]["end"] = ["r0", "r1"]
  runner = runner_for(d, dtype, 512, 8)
  got = rc.run_in_process(runner, trace)
  got = {k: v for k, v in got.items() if k[0] == "r0" or k[1] < pos_b}
  compare(got, ref, dtype, f"besolix long decode {tag}/{dtype}")
  runner.cache.check_invariants()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts_whole_and_in_large_portions(besolix_dirs, dtype):
  """Prompts of 1300 and 700 tokens, the first in one step, the second in portions of 600 and 100: the delta rule's walk of long
  portions, a dozen windows in one launch, the many-row products; what they leave carries on into single tokens."""
  d = besolix_dirs("C")
  reqs = rc.make_requests(plain.CONFIGS["C"]["vocab"], (1300, 700), seed=17)
  ref = reference(d, reqs)
  a, b = reqs["r0"], reqs["r1"]
  want = lambda lo, hi: list(range(0, hi - lo, 37)) + [hi - lo - 1]
  trace = [{"step": 0, "entries": [{"id": "r0", "tokens": a[:1290], "want": want(0, 1290)}], "end": []}]
  trace += [{"step": 1 + j, "entries": [{"id": "r0", "tokens": [a[1290 + j]], "want": [0]}], "end": ["r0"] if j == 9 else []} for j in range(10)]
  trace.append({"step": 11, "entries": [{"id": "r1", "tokens": b[:600], "want": want(0, 600)}], "end": []})
  trace.append({"step": 12, "entries": [{"id": "r1", "tokens": b[600:], "want": want(600, 700)}], "end": ["r1"]})
  runner = runner_for(d, dtype, 1344, 64)
  got = rc.run_in_process(runner, trace)
  compare(got, ref, dtype, f"besolix long prompts/{dtype}")
  runner.cache.check_invariants()
  runner.runner.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_slot_and_pages_that_are_used_again(besolix_dirs, dtype):
  """One request slot and its pages: six requests one after the other, each ended before the next comes, the third of them
  cut off in the middle of its prompt.  Every one finds its own keys only, whatever the pages held before."""
  d = besolix_dirs("A")
  reqs = rc.make_requests(plain.CONFIGS["A"]["vocab"], (40, 64, 50, 7, 33, 2), seed=12)
  ref = reference(d, reqs)
  runner = runner_for(d, dtype, 64, 16, max_requests=1)
  trace = []
  for rid, ids in reqs.items():
    if rid == "r2":                            # given up half way: what it wrote stays behind in slot and pages
      trace.append({"step": len(trace), "entries": [{"id": "x", "tokens": ids[:25], "want": []}], "end": ["x"]})
    cut = max(1, len(ids) // 3)
    trace.append({"step": len(trace), "entries": [{"id": rid, "tokens": ids[:cut], "want": list(range(cut))}], "end": []})
    if cut < len(ids):
      trace.append({"step": len(trace), "entries": [{"id": rid, "tokens": ids[cut:], "want": list(range(len(ids) - cut))}], "end": [rid]})
    else:
      trace[-1]["end"] = [rid]
  got = rc.run_in_process(runner, trace)
  got = {k: v for k, v in got.items() if k[0] != "x"}
  assert len(got) == sum(len(v) for v in reqs.values())
  compare(got, ref, dtype, f"besolix slots used again/{dtype}")
  runner.cache.check_invariants()
  assert runner.cache.free_pages() == [g.num_pages for g in runner.cache.paged_groups]


# Weights under which single keys stand out: the scores of a window's keys are spread over tens of units, so that a position's
# output is the values of a handful of keys, as often at a window's far edge as near.  A key outside the window, a wrong page
# or a wrong position moves the row as a whole (tests/test_besolix_cpu.py measures by how much).
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cut", ["whole", "tail", "portions"])
def test_single_keys_that_stand_out_in_prompts_and_in_decoding(tmp_path, dtype, cut):
  cfg, W = plain.peaky_model()
  d = plain.write_model(cfg, W, str(tmp_path / "peaky"))
  reqs = rc.make_requests(cfg["vocab"], (600, 333), seed=6)
  ref = reference(d, reqs)
  trace = {"whole": rc.whole, "tail": lambda r: rc.tail_one_by_one(r, 140), "portions": rc.portions}[cut](reqs)
  runner = runner_for(d, dtype, 640, 64)
  got = rc.run_in_process(runner, trace)
  if dtype == "float32":
    compare(got, ref, dtype, f"besolix peaky/{cut}")
  else:      # scores this sharp turn on roundings of queries and keys for single rows: most rows are held to the bound
    size = float(np.sqrt(np.mean([float(r.pow(2).mean()) for r in ref.values()])))
    errs = np.array([float(np.sqrt(((row - ref[k[0]][k[1]].numpy()) ** 2).mean())) / size for k, row in got.items()])
    assert np.isfinite(errs).all() and np.median(errs) <= 0.1 and (errs > 0.3).mean() <= 0.1, (np.median(errs), (errs > 0.3).mean())
  runner.cache.check_invariants()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["C", "E"])
def test_steps_of_one_shape_that_are_replayed(besolix_dirs, dtype, tag):
  """Five prompts of one length whole, one after the other, then their tails in portions of one size: from the second step of
  a shape on it is recorded and replayed, with other pages and other tokens each time."""
  d = besolix_dirs(tag)
  reqs = rc.make_requests(plain.CONFIGS[tag]["vocab"], (150,) * 5, seed=31)
  ref = reference(d, reqs)
  trace = []
  for rid, ids in reqs.items():
    for lo, hi in ((0, 100), (100, 125), (125, 150)):
      trace.append({"step": len(trace), "entries": [{"id": rid, "tokens": ids[lo:hi], "want": list(range(hi - lo))}], "end": [rid] if hi == 150 else []})
  runner = runner_for(d, dtype, 384, 64)
  got = rc.run_in_process(runner, trace)
  compare(got, ref, dtype, f"besolix replayed {tag}/{dtype}")
  assert DEV == "cpu" or runner.runner.num_graphs() >= 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_request_left_out_for_many_steps_goes_on_where_it_was(besolix_dirs, dtype):
  """One request pauses off a page's edge, while others come, end and leave their pages and slots; then it goes on with a
  portion of two tokens, and token by token over the ends of its windows."""
  d = besolix_dirs("C")
  reqs = rc.make_requests(plain.CONFIGS["C"]["vocab"], (230, 100, 64, 90), seed=23)
  ref = reference(d, reqs)
  ids = reqs["r0"]
  trace = [{"step": 0, "entries": [{"id": "r0", "tokens": ids[:151], "want": [0, 95, 96, 150]}], "end": []}]
  for rid in ("r1", "r2", "r3"):
    t = reqs[rid]
    trace.append({"step": len(trace), "entries": [{"id": rid, "tokens": t[:40], "want": [39]}], "end": []})
    trace.append({"step": len(trace), "entries": [{"id": rid, "tokens": t[40:], "want": list(range(len(t) - 40))}], "end": [rid]})
  trace.append({"step": len(trace), "entries": [{"id": "r0", "tokens": ids[151:153], "want": [0, 1]}], "end": []})
  for j in range(153, 230):
    trace.append({"step": len(trace), "entries": [{"id": "r0", "tokens": [ids[j]], "want": [0]}], "end": ["r0"] if j == 229 else []})
  runner = runner_for(d, dtype, 384, 64)
  got = rc.run_in_process(runner, trace)
  compare(got, ref, dtype, f"besolix paused/{dtype}")
  runner.cache.check_invariants()


@pytest.mark.skipif(DEV == "cpu", reason="a property of the CUDA kernels' order of sums, not of the CPU statements")
@pytest.mark.parametrize("tag", ["A", "B"])
def test_float32_logits_do_not_depend_on_the_cut(besolix_dirs, tag):
  """In float32 a position's logits come out the same to the last bit however the request was cut and whatever else was
  in the batch: every sum of the 32-bit path runs in an order that depends on the position alone."""
  d = besolix_dirs(tag)
  reqs = rc.make_requests(plain.CONFIGS[tag]["vocab"], (70, 33, 90, 41), seed=3)
  whole = rc.run_in_process(runner_for(d, "float32", 128, 16), rc.whole(reqs))
  for name, trace in (("portions", rc.portions(reqs)), ("mixed", rc.mixed(reqs, 224, seed=4, granule=16))):
    got = rc.run_in_process(runner_for(d, "float32", 224, 16), trace)
    for key, row in got.items():
      assert np.array_equal(row, whole[key[:2]]), f"{name}: request {key[0]} position {key[1]} differs in its bits"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tag", ["A", "C"])
def test_greedy_generation_through_the_engine(besolix_dirs, dtype, tag):
  """``LLMEngine.generate``: the scheduler admits, cuts the prompts into portions under a small token budget, decodes from
  CUDA graphs; more requests than slots, so state slots and pages are used again."""
  from miniinfer_b200 import LLMEngine, SamplingParams
  d = besolix_dirs(tag)
  W, cfg = plain.read_weights(d), plain.read_config(d)
  g = torch.Generator().manual_seed(21)
  prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (3, 45, 18, 70, 9, 31)]
  n_new = 40
  page = PAGES[tag]
  eng = LLMEngine(d, dtype=dtype, device=DEV, page_size=page, num_pages=3 * (128 // page), max_num_seqs=3, max_model_len=128,
                  max_num_batched_tokens=32)
  outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=n_new, ignore_eos=True))
  size = float(plain.forward(cfg, W, prompts[1]).pow(2).mean().sqrt())
  for prompt, out in zip(prompts, outs):
    ids = out["token_ids"]
    assert len(ids) == n_new
    # every token is the plain implementation's choice for the text so far, or within rounding of it
    seq, odd = list(prompt), 0
    for t in ids:
      row = plain.forward(cfg, W, seq)[-1]
      odd += float(row.max() - row[t]) > (1e-3 if dtype == "float32" else 2 * BF16_BOUND) * size
      seq.append(t)
    assert odd <= (0 if dtype == "float32" else 0.1 * n_new), f"{odd} of {n_new} tokens are not what the plain logits allow"
  if DEV != "cpu":
    eng.runner.check_status()
    assert eng.runner.num_graphs() > 0


@pytest.mark.skipif(DEV == "cpu", reason="the command line runs on a CUDA device")
def test_command_line_and_trace_program(besolix_dirs, tmp_path):
  """`main.py` generates from a Besolix folder, and `bin/trace_run` - a process of its own that picks the model by its
  configuration - replays a mixed trace in both dtypes."""
  import json
  import os
  import subprocess
  import sys
  root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
  d = besolix_dirs("B")
  W, cfg = plain.read_weights(d), plain.read_config(d)
  proc = subprocess.run([sys.executable, os.path.join(root, "main.py"), "--model", d, "--prompt-ids", "5,17,3,199", "--max-tokens", "6",
                         "--temperature", "0", "--dtype", "float32", "--max-model-len", "64", "--page-size", "16"],
                        capture_output=True, text=True, timeout=900)
  assert proc.returncode == 0, proc.stderr[-3000:]
  assert str(plain.generate(cfg, W, [5, 17, 3, 199], 6)) in proc.stdout
  reqs = rc.make_requests(cfg["vocab"], (70, 9, 130), seed=2)
  ref = reference(d, reqs)
  trace = rc.mixed(reqs, 256, seed=3)
  for dtype in ("float32", "bfloat16"):
    out = tmp_path / dtype
    proc = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out), "--max-tokens", "256"],
                          input="\n".join(json.dumps(r) for r in trace) + "\n", capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-3000:]
    assert [l for l in proc.stdout.split("\n") if l.startswith("done")] == [f"done {r['step']}" for r in trace]
    outputs = {r["step"]: np.fromfile(out / f"{r['step']}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
               for r in trace if sum(len(e["want"]) for e in r["entries"])}
    compare(rc.collect(trace, outputs), ref, dtype, f"trace program {dtype}")
