"""Each mechanism of the Korurax design alone: the engine's operation against the plain function of
tests/plain_korurax.py.  Inputs are made so that a fault shows: keys just inside and just outside a chunk whose scores stand
out, queries in several chunks of one tile, sizes that are no powers of two and values that a model may happen to make
equal or 1."""
import math

import pytest
import torch

import plain_korurax as plain
from gpu_helpers import DEV, make_attention_case

pytestmark = pytest.mark.gpu

DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def rounded(t, dtype):
  return t.to(DT[dtype]).float()


def plain_rows(qkv, kv, bt, batch, nh, nkv, hd, scale, chunk=None, sink=None, gate=None, r1=None, r2=None, out_hd=None):
  """Every row of the step from the cache, in float64, with the mechanisms that are given."""
  T, P, G = qkv.shape[0], kv.shape[3], nh // nkv
  q = qkv.double().view(T, -1, hd)[:, :nh]
  pos, item, slots = batch.positions.long().cpu(), batch.token_item.cpu(), batch.seq_slot.tolist()
  out = torch.zeros((T, nh, hd), dtype=torch.float64)
  for b, slot in enumerate(slots):
    rows = (item == b).nonzero()[:, 0]
    p = pos[rows]
    js = torch.arange(0, int(p.max()) + 1)
    pages = bt[slot].long()[js // P]
    k = kv[pages, 0, :, js % P, :].double().repeat_interleave(G, dim=1)
    v = kv[pages, 1, :, js % P, :].double().repeat_interleave(G, dim=1)
    seen = plain.same_chunk(len(js), chunk)[p]
    s = torch.einsum("thd,nhd->htn", q[rows], k) * scale
    if r1 is not None:
      s = s - plain.distance_bias(len(js), r1.double(), r2.double())[:, p]
    w = plain.softmax_with_sink(s, seen[None], sink.double() if sink is not None else None)
    out[rows] = torch.einsum("htn,nhd->thd", w, v)
  if gate is not None:
    out = out * torch.sigmoid(gate.double())[:, :, None]
  return out[:, :, :out_hd].reshape(T, -1).float()


CASES = [
  # (context, new tokens) of every request; heads, kv heads, head size, page size, chunk
  ([(300, 300), (77, 1), (1, 1), (129, 2)], 4, 2, 64, 64, 96),       # the tcgen05 prefill kernel; chunks' edges inside its tiles
  ([(500, 300), (257, 1), (129, 3)], 6, 2, 64, 64, 128),             # three query heads a kv head; chunks that are the tiles
  ([(200, 1), (64, 1), (65, 1), (1000, 1)], 8, 2, 64, 64, 120),      # decode tokens only: the cluster kernel
  ([(900, 1)] * 40, 8, 4, 64, 64, 800),                              # more than fit at once: the persistent kernel
  ([(130, 67), (40, 1), (16, 16), (17, 1)], 6, 1, 48, 16, 20),       # heads of 48, pages of 16: the mma.sync prefill and the cp.async decode kernel
  ([(90, 1), (33, 33)], 3, 3, 24, 8, 7),                             # heads of 24: the generic kernel in both dtypes
  ([(300, 300), (77, 1), (700, 1), (129, 2)], 8, 1, 128, 64, 250),   # heads of 128, eight query heads on one kv head
  ([(130, 67), (40, 1), (300, 1)], 2, 1, 256, 64, 64),               # heads of 256, chunks that are pages
  ([(150, 150), (65, 1), (64, 1)], 10, 5, 80, 16, 1),                # chunks of one token: everybody sees himself
  ([(520, 1), (64, 1), (70, 66)], 32, 2, 64, 64, 333),               # sixteen query heads on a kv head
  ([(70, 70), (33, 1), (40, 2)], 3, 1, 272, 16, 24),                 # rows of more than 256 values: no tensor cores
]


def options(case, nh, seed=0):
  g = torch.Generator().manual_seed(1000 + case + seed)
  r1 = 0.2 + 1.5 * torch.rand(nh, generator=g)
  r2 = torch.exp(-1.5 + torch.randn(nh, generator=g))
  return r1, r2, 1.0 + torch.randn(nh, generator=g)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", range(len(CASES)))
@pytest.mark.parametrize("which", ["all", "chunk", "distance", "gate", "narrow"])
def test_chunks_distance_and_gates_in_every_attention_kernel(dtype, case, which):
  """Prompts' portions and single tokens in one step: everything at once, then each mechanism alone, then all of them with
  output heads narrower than the cache rows."""
  from miniinfer_b200.kernels import ops
  items, nh, nkv, hd, page, chunk = CASES[case]
  if which != "all" and len(items) > 10:
    items = items[:10]
  qkv, kv, bt, batch = make_attention_case(items, nh, nkv, hd, page, DT[dtype], seed=case, scale_q=1.5, num_slots=64)
  r1, r2, sink = options(case, nh)
  T = qkv.shape[0]
  width, off = 3 + nh + 2, 3                                          # gate logits somewhere in wider rows, at an odd place
  rows = rounded(torch.randn((T, width), generator=torch.Generator().manual_seed(case)) * 2.0, dtype)
  gate = rows[:, off:off + nh]
  scale = 1.3 / math.sqrt(hd)
  every = which in ("all", "narrow")
  ohd = hd - hd // 4 if which == "narrow" else hd
  kw, pk = {}, {}
  if every or which == "chunk":
    kw["chunk"] = pk["chunk"] = chunk
  if every or which == "distance":
    kw["distance"] = torch.cat((r1, r2)).to(DEV)
    pk.update(r1=r1, r2=r2)
  if every or which == "gate":
    kw.update(gate=rows.to(DT[dtype]).to(DEV), gate_offset=off, gate_per_head=True)
    pk["gate"] = gate
  if every:
    kw["sink"] = sink.to(DEV)
    pk["sink"] = sink
  out = torch.zeros((T, nh * ohd), dtype=DT[dtype], device=DEV)
  ops.attention(out, qkv, kv, bt, batch, nh, nkv, hd, scale, None, out_hd=ohd, **kw)
  want = plain_rows(qkv.cpu(), kv.cpu(), bt.cpu(), batch, nh, nkv, hd, scale, out_hd=ohd, **pk)
  assert float((out.float().cpu() - want).abs().max()) <= (2e-5 if dtype == "float32" else 1.5e-2) * float(want.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hd,page,nh,nkv", [(64, 64, 4, 2), (48, 16, 6, 1), (128, 64, 3, 1), (32, 64, 2, 2)])
@pytest.mark.parametrize("chunk", [64, 96, 130])
def test_keys_on_both_sides_of_every_chunks_edge(dtype, hd, page, nh, nkv, chunk):
  """The last key of a chunk and the first of the next have scores that no other key comes near: a token right behind the
  edge must return the first key's value and nothing of the last one's, the tokens before it the reverse; portions that
  start at the edge, one before it and one behind it, and single tokens there."""
  from miniinfer_b200.kernels import ops
  edges = [chunk * i for i in range(1, 400 // chunk + 1)]
  for ctx, new in [(400, 400), (edges[0] + 2, 3), (edges[-1] + 1, 2), (edges[0], 1), (edges[0] + 1, 1), (edges[-1] + 2, 1)]:
    qkv, kv, bt, batch = make_attention_case([(ctx, new)], nh, nkv, hd, page, DT[dtype], seed=ctx, scale_q=0.01)
    slot = int(batch.seq_slot[0])
    mark = torch.ones(hd) / math.sqrt(hd)
    T = qkv.shape[0]
    qkv.view(T, -1, hd)[:, :nh] += (30.0 * mark).to(DT[dtype]).to(DEV)                 # every query looks for the mark ...
    kv[:, 0] = 0
    for j in [x for e in edges for x in (e - 1, e) if x < ctx]:
      kv[bt[slot, j // page].long(), 0, :, j % page] = (mark * 4.0).to(DT[dtype]).to(DEV)   # ... which only the keys at the edges carry
    out = torch.zeros((T, nh * hd), dtype=DT[dtype], device=DEV)
    r1, r2 = torch.full((nh,), 0.5), torch.full((nh,), 0.25)
    ops.attention(out, qkv, kv, bt, batch, nh, nkv, hd, 1.0, None, chunk=chunk, distance=torch.cat((r1, r2)).to(DEV))
    want = plain_rows(qkv.cpu(), kv.cpu(), bt.cpu(), batch, nh, nkv, hd, 1.0, chunk=chunk, r1=r1, r2=r2)
    assert float((out.float().cpu() - want).abs().max()) <= (1e-4 if dtype == "float32" else 3e-2) * float(want.abs().max()), (ctx, new)
    # the token at an edge sees that key alone
    for t in range(T):
      p = int(batch.positions[t])
      if p in edges:
        v = kv[bt[slot, p // page].long(), 1, :, p % page].float().repeat_interleave(nh // nkv, 0)
        assert float((out[t].float().view(nh, hd) - v).abs().max()) <= (1e-5 if dtype == "float32" else 2e-2) * float(v.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_pays_for_its_distance(dtype):
  """One key stands out 900 positions back in a chunk of 1000: with r1 = 0 the output is its value; with a distance bias
  that costs more than its score it is as if it were not there; the sink takes what is left."""
  from miniinfer_b200.kernels import ops
  nh, nkv, hd, page, far = 4, 2, 64, 64, 100
  for items in ([(1000, 1)], [(1000, 100)]):
    qkv, kv, bt, batch = make_attention_case(items, nh, nkv, hd, page, DT[dtype], seed=5, scale_q=0.02)
    slot = int(batch.seq_slot[0])
    key = kv[bt[slot, far // page].long(), 0, :, far % page].float()
    for h in range(nh):
      qkv[-1, h * hd:(h + 1) * hd] = (key[h // 2] * (25.0 / float(key[h // 2].pow(2).sum()))).to(DT[dtype])      # a score of 25
    value = kv[bt[slot, far // page].long(), 1, :, far % page].float()
    r1 = torch.tensor([0.0, 2.0, 0.0, 8.0])
    r2 = torch.tensor([1.0, 0.5, 0.3, 0.5])
    sink = torch.tensor([-30.0, -30.0, 40.0, -30.0])
    out = torch.zeros((qkv.shape[0], nh * hd), dtype=DT[dtype], device=DEV)
    ops.attention(out, qkv, kv, bt, batch, nh, nkv, hd, 1.0, None, chunk=1000, distance=torch.cat((r1, r2)).to(DEV), sink=sink.to(DEV))
    got = out[-1].float().view(nh, hd)
    top = float(value.abs().max())
    assert float((got[0] - value[0]).abs().max()) <= 0.05 * top            # nothing is paid
    assert float((got[1] - value[0]).abs().max()) <= 0.1 * top             # 25 - 2 ln 451 is still far above the rest
    assert float(got[2].abs().max()) <= 0.05 * top                         # the sink outbids the key
    assert float((got[3] - value[1]).abs().max()) > 0.3 * top              # 25 - 8 ln 451 < 0: the key is lost in the distance
    want = plain_rows(qkv.cpu(), kv.cpu(), bt.cpu(), batch, nh, nkv, hd, 1.0, chunk=1000, r1=r1, r2=r2, sink=sink)
    assert float((out.float().cpu() - want).abs().max()) <= (5e-5 if dtype == "float32" else 2e-2) * float(want.abs().max())


@pytest.mark.skipif(DEV == "cpu", reason="two forms of the CUDA kernel")
@pytest.mark.parametrize("chunk", [None, 150, 256])
def test_distance_bias_with_blocks_in_pairs(chunk, monkeypatch):
  """The tcgen05 prefill kernel with two blocks on a work (what steps of thousands of new tokens take): the rows of blocks
  that work alone, and the plain sums."""
  from miniinfer_b200.kernels import ops
  nh, nkv, hd, page = 8, 2, 128, 64
  qkv, kv, bt, batch = make_attention_case([(400, 400), (129, 2), (64, 1)], nh, nkv, hd, page, torch.bfloat16, seed=9, scale_q=1.5)
  r1, r2, sink = options(99, nh)
  rows = torch.randn((qkv.shape[0], nh), generator=torch.Generator().manual_seed(2)).to(torch.bfloat16)
  outs = []
  for pairs in ("1", "0"):
    monkeypatch.setenv("MINIINFER_B200_PREFILL_PAIRS", pairs)
    out = torch.zeros((qkv.shape[0], nh * hd), dtype=torch.bfloat16, device=DEV)
    ops.attention(out, qkv, kv, bt, batch, nh, nkv, hd, hd ** -0.5, None, chunk=chunk, distance=torch.cat((r1, r2)).to(DEV), sink=sink.to(DEV),
                  gate=rows.to(DEV), gate_per_head=True)
    outs.append(out.float().cpu())
  want = plain_rows(qkv.cpu(), kv.cpu(), bt.cpu(), batch, nh, nkv, hd, hd ** -0.5, chunk=chunk, r1=r1, r2=r2, sink=sink, gate=rows.float())
  for o in outs:
    assert float((o - want).abs().max()) <= 1.5e-2 * float(want.abs().max())
  assert float((outs[0] - outs[1]).abs().max()) <= 4e-3 * float(want.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W", [24, 65, 320, 1000, 4096, 5000])
@pytest.mark.parametrize("kind", ["layer", "rms", None])
def test_a_step_of_the_residual_stream(dtype, W, kind):
  """X = x + mult y, kept; the average over 0, 1, 6 and 9 earlier layers beside the embedding's rows; the norm of it - all rows
  and selected ones, in place and not, with and without a bias, without a sublayer's output."""
  from miniinfer_b200.kernels import ops
  g = torch.Generator().manual_seed(W)
  T, mult, eps = 7, 0.7, 1e-5
  x, first = torch.randn((T, W), generator=g) * 2.0 + 0.5, torch.randn((T, W), generator=g)
  later = torch.randn((9, T, W), generator=g)
  y = rounded(torch.randn((T, W), generator=g), dtype)
  w, b = 1.0 + 0.3 * torch.randn(W, generator=g), torch.randn(W, generator=g)
  rows = torch.tensor([5, 0, 5, 3], dtype=torch.int32)
  dev = lambda t: t.to(DEV)
  X = x.double() + mult * y.double()
  for n, with_y, with_b, pick in ((None, True, False, False), (None, False, True, False), (0, True, False, False), (1, True, True, True),
                                  (6, True, False, True), (6, False, False, False), (9, True, False, False)):
    Xn = X if with_y else x.double()
    wts = None if n is None else torch.randn(n + 2, generator=g) * 3.0
    v = Xn if n is None else plain.depth_average([first.double()] + [l.double() for l in later[:n]] + [Xn], wts.double())
    norm = {"layer": plain.layer_norm, "rms": plain.rms_norm}.get(kind)
    want = None if norm is None else norm(v, w.double(), eps) + (b.double() if with_b else 0.0)
    if pick and want is not None:
      want = want[rows.long()]
    xd, keep = dev(x.clone()), torch.zeros((T, W), device=DEV)
    x_out = None if (pick and kind) else (xd if n != 1 else torch.zeros((T, W), device=DEV))
    out = torch.zeros((4 if pick else T, W), dtype=DT[dtype], device=DEV) if kind else None
    ops.residual_step(out, xd, dev(y).to(DT[dtype]) if with_y else None, mult, x_out,
                      (kind, dev(w), dev(b) if with_b else None, eps) if kind else None, dev(rows) if (pick and kind) else None,
                      weights=dev(wts) if wts is not None else None, first=dev(first) if wts is not None else None,
                      later=dev(later) if n else None, n_later=n or 0, keep=keep if n not in (None, 9) and not pick else None)
    top = float(v.abs().max())
    if x_out is not None:
      assert float((x_out.double().cpu() - v).abs().max()) <= 2e-6 * max(top, 1.0), (n, with_y)
    if n not in (None, 9) and not pick:
      assert float((keep.double().cpu() - Xn).abs().max()) <= 1e-6 * float(Xn.abs().max())
    else:
      assert float(keep.abs().max()) == 0
    if want is not None:
      assert float((out.double().cpu() - want).abs().max()) <= (2e-5 if dtype == "float32" else 1e-2) * float(want.abs().max()), (n, with_y, pick)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W", [40, 65, 1024])
def test_layer_norm_without_a_bias(dtype, W):
  from miniinfer_b200.kernels import ops
  g = torch.Generator().manual_seed(W)
  x, d = torch.randn((5, W), generator=g) + 3.0, rounded(torch.randn((5, W), generator=g), dtype)
  w = 1.0 + 0.3 * torch.randn(W, generator=g)
  out = torch.zeros((5, W), dtype=DT[dtype], device=DEV)
  xd = x.clone().to(DEV)
  ops.add_layernorm(out, xd, d.to(DT[dtype]).to(DEV), None, w.to(DEV), None, 1e-3, None, True)
  want = plain.layer_norm(x.double() + d.double(), w.double(), 1e-3).float()
  assert float((out.float().cpu() - want).abs().max()) <= (2e-5 if dtype == "float32" else 1e-2) * float(want.abs().max())
  assert float((xd.cpu() - (x + d)).abs().max()) <= 1e-6


@pytest.mark.parametrize("n,cap", [(1, 30.0), (37, 4.0), (4099, 1.0), (100003, 25.0)])
def test_capped_logits(n, cap):
  from miniinfer_b200.kernels import ops
  x = torch.randn(n, generator=torch.Generator().manual_seed(n)) * 2.0 * cap
  xd = x.clone().to(DEV)
  ops.softcap(xd, cap)
  assert float((xd.double().cpu() - cap * torch.tanh(x.double() / cap)).abs().max()) <= 2e-6 * cap


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,E,top,H,F", [(1, 5, 2, 64, 24), (7, 3, 3, 32, 16), (16, 40, 6, 1032, 40), (70, 4, 1, 64, 40), (700, 4, 2, 128, 64),
                                          (1800, 6, 2, 64, 96)])
def test_squared_relu_experts_by_scaled_sigmoid_shares(dtype, T, E, top, H, F):
  """The largest sigmoid scores choose, their shares times a constant weigh, an expert is down(relu(up x)^2): few rows, many
  rows (the tcgen05 grouped product in bfloat16), all experts chosen, one chosen (whose share is the constant itself)."""
  from miniinfer_b200.engine.context import Workspace
  from miniinfer_b200.kernels import ops
  g = torch.Generator().manual_seed(T + E)
  W = {"m.router": rounded(torch.randn((E, H), generator=g) * 2.5 / math.sqrt(H), dtype)}
  for e in range(E):
    W[f"m.e{e}.up"] = rounded(torch.randn((F, H), generator=g) / math.sqrt(H), dtype)
    W[f"m.e{e}.down"] = rounded(torch.randn((H, F), generator=g) / math.sqrt(F), dtype)
  x = rounded(torch.randn((T, H), generator=g), dtype)
  mlp = plain.moe(F, E, top, 1.7)
  want = plain.mixture(x.double(), {k: v.double() for k, v in W.items()}, "m.", mlp).float()
  s = torch.sort(x.double() @ W["m.router"].double().T, dim=-1, descending=True).values
  clear = (s[:, top - 1] - s[:, top]) > (1e-4 if dtype == "float32" else 0.02) if top < E else torch.ones(T, dtype=torch.bool)
  dev = lambda t: t.to(DT[dtype]).to(DEV)
  out = torch.zeros((T, H), dtype=DT[dtype], device=DEV)
  ops.routed_experts(out, dev(x), dev(W["m.router"]), None, dev(torch.stack([W[f"m.e{e}.up"] for e in range(E)])),
                     dev(torch.stack([W[f"m.e{e}.down"] for e in range(E)])), top, Workspace(torch.device(DEV)), glu="relu_squared", weight_scale=1.7)
  diff = (out.float().cpu() - want).abs().max(-1).values
  assert int(clear.sum()) >= 0.8 * T
  assert float(diff[clear].max()) <= (3e-5 if dtype == "float32" else 3e-2) * float(want.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,ff,W", [(1, 24, 64), (9, 40, 72), (40, 96, 128), (2000, 64, 128)])
def test_clamped_dense_feed_forward(dtype, T, ff, W):
  """The part itself, its limit small enough to bite: a few rows, a few dozen, thousands (the tcgen05 product)."""
  from types import SimpleNamespace
  from miniinfer_b200.engine.context import Workspace
  from miniinfer_b200.parts import SwiGLUFeedForward
  g = torch.Generator().manual_seed(T)
  P = {k: rounded(torch.randn(s, generator=g) * f / math.sqrt(s[1]), dtype)
       for k, s, f in (("gate", (ff, W), 2.0), ("up", (ff, W), 2.0), ("down", (W, ff), 1.0))}
  part = SwiGLUFeedForward("m", W, ff, tensors=("gate", "up", "down"), activation="clamped", limit=0.6)
  dev = lambda t: t.to(DT[dtype]).to(DEV)
  part.bind({"gate_up": dev(torch.cat((P["gate"], P["up"]))), "down": dev(P["down"])})
  x = rounded(torch.randn((T, W), generator=g), dtype)
  got = part.forward(dev(x), SimpleNamespace(ws=Workspace(torch.device(DEV)), dtype=DT[dtype]))
  want = plain.clamped_glu(x.double(), {"m." + k: v.double() for k, v in P.items()}, "m.", 0.6).float()
  assert float((got.float().cpu() - want).abs().max()) <= (3e-5 if dtype == "float32" else 3e-2) * float(want.abs().max())
