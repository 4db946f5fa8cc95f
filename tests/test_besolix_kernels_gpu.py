"""Each mechanism of the Besolix design alone: the engine's operation, run over a step cut in several ways, against the plain
function of tests/plain_besolix.py on the whole sequence.  Inputs are made so that a fault shows: one key whose score stands
out just inside or just outside a window; states that must survive a cut; decays of nothing and of everything; sizes that are
no powers of two and values that a model may happen to make equal or 1."""
import math
from types import SimpleNamespace

import pytest
import torch

import plain_besolix as plain
from gpu_helpers import DEV, make_attention_case

pytestmark = pytest.mark.gpu

DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def tol(dtype):
  return 3e-5 if dtype == "float32" else 4e-2


def rounded(t, dtype):
  return t.to(DT[dtype]).double()


def workspace():
  from miniinfer_b200.engine.context import Workspace
  return Workspace(torch.device(DEV))


# ------------------------------------------------------------------------------------------ the delta rule


class DeltaCase:
  """Inputs of a gated delta rule with one decay a head and what the plain recurrence makes of them."""

  def __init__(self, T, H, G, D, Dv, dtype, seed=0, shift=-1.5, eps=1e-5):
    g = torch.Generator().manual_seed(1000 * H + D + Dv + seed)
    r = lambda *s: torch.randn(s, generator=g)
    self.sizes, self.T, self.dtype, self.eps = (H, G, D, Dv), T, dtype, eps
    # rows as the fused projection leaves them: gate | q | k | v | beta's logits | decays' logits, a few columns beyond
    self.widths = (H * Dv, G * D, G * D, H * Dv, H, H)
    self.rows = r(T, sum(self.widths) + 3).to(DT[dtype])
    self.dt_bias, self.A_log, self.norm = r(H) + shift, torch.rand((H,), generator=g) - 0.5, 1 + 0.1 * r(Dv)

  def columns(self, rows):
    out, at = [], 0
    for w in self.widths:
      out.append(rows[:, at:at + w])
      at += w
    return out

  def want(self):
    """(rows [T, H * Dv], the state [H, D, Dv] behind them)."""
    H, G, D, Dv = self.sizes
    T = self.T
    gate, q, k, v, b, a = self.columns(self.rows.double())
    q = (plain.unit(q.view(T, G, D)) * D ** -0.5).repeat_interleave(H // G, 1)
    k = plain.unit(k.view(T, G, D)).repeat_interleave(H // G, 1)
    decay = torch.exp(-torch.exp(self.A_log.double()) * torch.nn.functional.softplus(a + self.dt_bias.double()))
    beta = torch.sigmoid(b)
    o = plain.delta_rule(q, k, v.view(T, H, Dv), decay, beta)
    S = torch.zeros(H, D, Dv, dtype=torch.float64)
    for t in range(T):
      S = decay[t][:, None, None] * S
      S = S + torch.einsum("hd,hv->hdv", k[t], beta[t][:, None] * (v.view(T, H, Dv)[t] - torch.einsum("hdv,hd->hv", S, k[t])))
    return (plain.rms(o, self.eps) * self.norm.double() * plain.silu(gate.view(T, H, Dv))).reshape(T, -1), S

  def run(self, state, lo, hi, others=(), slot=2, ws=None):
    """Tokens lo..hi of the request in ``slot``, beside ``others`` = [(slot, lo, hi), ...] of the same rows; -> this request's rows."""
    from miniinfer_b200.kernels import ops
    H, G, D, Dv = self.sizes
    spans = [(slot, lo, hi)] + list(others)
    rows = torch.cat([self.rows[a:b] for _, a, b in spans]).to(DEV)
    q_len = [b - a for _, a, b in spans]
    dev = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    ctx = SimpleNamespace(q_start=dev([sum(q_len[:i]) for i in range(len(q_len))]), q_len=dev(q_len), seq_slot=dev([s for s, _, _ in spans]),
                          num_items=len(q_len), num_tokens=sum(q_len), token_item=dev([i for i, n in enumerate(q_len) for _ in range(n)]))
    gate, q, k, v, b, a = self.columns(rows)
    out = torch.zeros((rows.shape[0], H * Dv), dtype=DT[self.dtype], device=DEV)
    ops.gated_delta(out, q, k, v, a, b, gate, self.dt_bias.to(DEV), self.A_log.to(DEV), self.norm.to(DEV), self.eps, state, ctx, H, G, D, Dv,
                    workspace=ws, gate_silu=True)
    return out[:hi - lo].double().cpu()


def cuts_of(T, sizes):
  out, pos, k = [], 0, 0
  while pos < T:
    n = min(sizes[k % len(sizes)], T - pos)
    out.append((pos, pos + n))
    pos += n
    k += 1
  return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,Dv", [(2, 1, 16, 24), (4, 4, 32, 48), (3, 1, 8, 40), (2, 2, 64, 64), (1, 1, 128, 128), (2, 1, 40, 8), (6, 3, 96, 33),
                                      (1, 1, 1, 1), (2, 1, 10, 6), (3, 3, 200, 17)])
def test_delta_rule_with_one_decay_a_head(dtype, H, G, D, Dv):
  T = 45
  c = DeltaCase(T, H, G, D, Dv, dtype)
  want, last = c.want()
  bound = tol(dtype) * max(1.0, float(want.abs().max()))
  for sizes in ((T,), (1,), (2, 7, 1, 33), (2,)):
    state = torch.zeros((4, H * D * Dv + 3), dtype=torch.float32, device=DEV)
    got = torch.cat([c.run(state, a, b) for a, b in cuts_of(T, sizes)])
    assert float((got - want).abs().max()) <= bound, f"cut into {sizes}"
    assert float((state[2, :H * D * Dv].double().cpu().view(H, D, Dv) - last).abs().max()) <= 3e-5 * max(1.0, float(last.abs().max()))
    assert not state[[0, 1, 3]].any() and not state[2, H * D * Dv:].any()      # other slots, and what lies behind the state, untouched


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,Dv", [(2, 1, 24, 40), (1, 1, 128, 64), (4, 2, 64, 128), (3, 3, 50, 20), (16, 8, 32, 32)])
def test_delta_rule_of_long_portions(dtype, H, G, D, Dv):
  """Portions of hundreds of tokens, also beside single tokens and short portions of other requests: the result is the
  recurrence's whatever way the kernels walk it, and the state left behind lets the request go on token by token."""
  T = 1300
  c = DeltaCase(T, H, G, D, Dv, dtype, shift=-3.0)
  want, last = c.want()
  bound = 2 * tol(dtype) * max(1.0, float(want.abs().max()) / 4)
  for cuts in ((600, 2, 690, 1, 1, 1, 1, 1, 1, 1, 1), (1290,) + (1,) * 10, (520, 780), (63, 64, 159, 160, 161, 128, 192, 373)):
    for others in ((), ((0, 0, 1), (1, 0, 37), (3, 10, 12))):
      state = torch.zeros((4, H * D * Dv), dtype=torch.float32, device=DEV)
      got, pos = [], 0
      for n in cuts:
        got.append(c.run(state, pos, pos + n, others=others))
        pos += n
      assert pos == T
      assert float((torch.cat(got) - want).abs().max()) <= bound, f"cut into {cuts}, beside {others}"
      assert float((state[2].double().cpu().view(H, D, Dv) - last).abs().max()) <= 2e-3 * max(1.0, float(last.abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T", [40, 700])
@pytest.mark.parametrize("what", ["keeps everything", "forgets everything", "one head each", "a burst of forgetting"])
def test_extreme_decays(dtype, T, what):
  """Decays of 1 and of 0 (also underflowing ones) and both side by side: what was written long ago is there in full or not at all."""
  H, G, D, Dv = 2, 1, 32, 48
  c = DeltaCase(T, H, G, D, Dv, dtype)
  c.rows[:, -3 - H:-3] = 0.0                                  # the decays' logits: the bias decides
  if what == "keeps everything":
    c.dt_bias = torch.full((H,), -40.0)
  elif what == "forgets everything":
    c.dt_bias, c.A_log = torch.full((H,), 30.0), torch.full((H,), 3.0)
  elif what == "one head each":
    c.dt_bias, c.A_log = torch.tensor([-40.0, 30.0]), torch.tensor([0.0, 3.0])
  else:
    c.dt_bias = torch.full((H,), -8.0)
    c.rows[T // 2, -3 - H:-3] = 200.0
    c.A_log = torch.full((H,), 1.0)
  # early keys come back as late queries, so that the memory of them matters
  gate, q, k, v, b, a = c.columns(c.rows)
  q[T // 2:] = k[:T - T // 2]
  want, last = c.want()
  bound = 2 * tol(dtype) * max(1.0, float(want.abs().max()))
  for sizes in ((T,), (T - 3, 1, 2)):
    state = torch.zeros((4, H * D * Dv), dtype=torch.float32, device=DEV)
    got = torch.cat([c.run(state, x, y) for x, y in cuts_of(T, sizes)])
    assert torch.isfinite(got).all() and float((got - want).abs().max()) <= bound, f"cut into {sizes}"
    assert float((state[2].double().cpu().view(H, D, Dv) - last).abs().max()) <= 1e-4 * max(1.0, float(last.abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_keys_that_repeat_in_long_portions(dtype):
  """Every token writes along one of two nearly equal keys with beta near 1: each write corrects the one before it, which a walk
  that treats a stretch of tokens at once has to resolve exactly."""
  T, H, G, D, Dv = 640, 2, 1, 48, 32
  c = DeltaCase(T, H, G, D, Dv, dtype, shift=-6.0)
  gate, q, k, v, b, a = c.columns(c.rows)
  k[0::2] = k[0]
  k[1::2] = k[0] + 0.05 * k[1]
  b[:] = 5.0
  want, last = c.want()
  state = torch.zeros((4, H * D * Dv), dtype=torch.float32, device=DEV)
  got = torch.cat([c.run(state, x, y) for x, y in cuts_of(T, (600, 40))])
  assert float((got - want).abs().max()) <= 2 * tol(dtype) * max(1.0, float(want.abs().max()))


def test_float32_states_do_not_depend_on_the_cut():
  if DEV == "cpu":
    pytest.skip("a property of the CUDA kernels' order of sums")
  H, G, D, Dv, T = 4, 2, 48, 32, 700
  c = DeltaCase(T, H, G, D, Dv, "float32")
  runs = []
  for sizes in ((T,), (1, 2, 64, 65), (300, 3)):
    state = torch.zeros((4, H * D * Dv), dtype=torch.float32, device=DEV)
    runs.append((torch.cat([c.run(state, x, y) for x, y in cuts_of(T, sizes)]), state[2].cpu()))
  assert all(torch.equal(r[0], runs[0][0]) and torch.equal(r[1], runs[0][1]) for r in runs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("taps", [1, 2, 3, 6])
def test_short_convolutions_without_bias(dtype, taps):
  from miniinfer_b200.kernels import ops
  g = torch.Generator().manual_seed(taps)
  C, T = 56, 41
  x, w = torch.randn((T, C + 8), generator=g).to(DT[dtype]), torch.randn((C, taps), generator=g)
  want = plain.silu(plain.short_conv(x[:, 3:3 + C].double(), w.double()))
  for sizes in ((T,), (1,), (2,), (taps, 1, 5)):
    state = torch.zeros((3, max(1, (taps - 1) * C)), dtype=torch.float32, device=DEV)
    got = []
    for a, b in cuts_of(T, sizes):
      dev = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
      ctx = SimpleNamespace(q_start=dev([0]), q_len=dev([b - a]), seq_slot=dev([1]), num_items=1, token_item=dev([0] * (b - a)))
      out = torch.zeros((b - a, C), dtype=DT[dtype], device=DEV)
      ops.causal_conv(out, x[a:b].to(DEV)[:, 3:3 + C], w.to(DEV), None, state, ctx, silu=True)
      got.append(out.double().cpu())
    assert float((torch.cat(got) - want).abs().max()) <= tol(dtype), f"cut into {sizes}"


# ------------------------------------------------------------------------------------------ feed-forward, gates


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M,K,I", [(1, 64, 40), (3, 96, 200), (16, 128, 72), (17, 64, 24), (70, 72, 136), (1900, 128, 96)])
def test_tanh_gelu_gated_products(dtype, M, K, I):
  """From one row to many: the few-row product, the product with the activation kernel behind it, the tcgen05 product."""
  from miniinfer_b200.kernels import ops
  g = torch.Generator().manual_seed(M + K)
  x, w = torch.randn((M, K), generator=g).to(DT[dtype]), (2.0 * torch.randn((2 * I, K), generator=g) / math.sqrt(K)).to(DT[dtype])
  x[0] *= 12.0                                                # gates far out on both sides
  z = x.double() @ w.double().T
  zr = rounded(z, dtype)                                      # the products are rounded before the activation
  want = plain.gelu_tanh(zr[:, :I]) * zr[:, I:]
  outs = []
  for kw in ({}, {"force_stream": True}) if dtype == "bfloat16" and M <= 16 and K >= 64 and DEV != "cpu" else ({},):
    out = torch.zeros((M, I), dtype=DT[dtype], device=DEV)
    ops.linear_glu(out, x.to(DEV), w.to(DEV), workspace(), "gelu_tanh", **kw)
    outs.append(out.double().cpu())
  gu = zr.to(DT[dtype]).to(DEV)
  out = torch.zeros((M, I), dtype=DT[dtype], device=DEV)
  ops.glu_mul(out, gu, "gelu_tanh")
  outs.append(out.double().cpu())
  for o in outs:
    err = (o - want).abs()
    assert torch.isfinite(o).all() and float((err - tol(dtype) * want.abs()).max()) <= tol(dtype) * 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T", [3, 40, 900])
def test_tanh_gelu_gated_experts(dtype, T):
  from miniinfer_b200.kernels import ops
  g = torch.Generator().manual_seed(T)
  H, F, E, top = 64, 72, 4, 2
  x, router = torch.randn((T, H), generator=g).to(DT[dtype]), torch.randn((E, H), generator=g).to(DT[dtype])
  gu, dn = (torch.randn((E, 2 * F, H), generator=g) / 8).to(DT[dtype]), (torch.randn((E, H, F), generator=g) / 8).to(DT[dtype])
  out = torch.zeros((T, H), dtype=DT[dtype], device=DEV)
  ops.routed_experts(out, x.to(DEV), router.to(DEV), None, gu.to(DEV), dn.to(DEV), top, workspace(), weights="softmax_chosen", glu="gelu_tanh")
  z = x.double() @ router.double().T
  ch = torch.topk(z, top, -1)
  wt = torch.softmax(ch.values, -1)
  want = torch.zeros((T, H), dtype=torch.float64)
  for e in range(E):
    act = rounded(plain.gelu_tanh(x.double() @ gu[e, :F].double().T) * (x.double() @ gu[e, F:].double().T), dtype)
    want += (wt * (ch.indices == e)).sum(-1, keepdim=True) * (act @ dn[e].double().T)
  assert float((out.double().cpu() - want).abs().max()) <= tol(dtype) * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M,B,N,K,odd", [(1, 4, 24, 40, 0), (5, 3, 20, 12, 1), (16, 2, 64, 64, 0), (70, 2, 65, 33, 0), (40, 1, 32, 48, 0), (200, 6, 32, 64, 0),
                                         (33, 4, 16, 24, 3)])
def test_batched_product_with_a_gate_a_value(dtype, M, B, N, K, odd):
  from miniinfer_b200.kernels import ops
  g = torch.Generator().manual_seed(M + N)
  x, w = torch.randn((M, B * K), generator=g).to(DT[dtype]), (torch.randn((B, N, K), generator=g) / math.sqrt(K)).to(DT[dtype])
  rows = (3.0 * torch.randn((M, 16 + odd + B * N), generator=g)).to(DT[dtype])
  gate = rows[:, 16 + odd:]                                   # columns of wider rows, at an odd place too
  out = torch.zeros((M, B * N), dtype=DT[dtype], device=DEV)
  ops.linear_batched(out.view(M, B, N), x.to(DEV).view(M, B, K), w.to(DEV), value_gate=rows.to(DEV)[:, 16 + odd:])
  want = torch.einsum("mbk,bnk->mbn", x.view(M, B, K).double(), w.double()).reshape(M, -1) * torch.sigmoid(gate.double())
  assert float((out.double().cpu() - want).abs().max()) <= tol(dtype)


# ------------------------------------------------------------------------------------------ attention


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,R,Dv,C,Q,window", [(2, 16, 8, 24, 32, 40, 20), (3, 24, 16, 16, 48, 24, 1), (4, 32, 32, 64, 96, 64, 33), (1, 8, 2, 8, 16, 8, None),
                                                 (2, 16, 8, 24, 264, 40, 17)])
def test_latent_attention_with_a_window_a_value_gate_and_a_reader(dtype, H, D, R, Dv, C, Q, window):
  """Two layers over one cache, put together from the engine's operations: the first stores its latents, the second - with
  another window, more heads, weights of its own and no key/value row in its projection - reads them.  Both give what the plain
  formulas give with per-head keys and values, in a prompt's portions and decoding."""
  from miniinfer_b200.cache.manager import LayerCache
  from miniinfer_b200.parts import LatentAttentionMixer, LinearScaledRotaryEncoding
  from miniinfer_b200.parts.mixer import DecodeItems, PrefillTiles, PrefillWideTiles
  g = torch.Generator().manual_seed(C + R)
  T, page, eps, base, W = 50, 16, 1e-5, 5000.0, 48
  r = lambda *s: torch.randn(s, generator=g)
  pe = LinearScaledRotaryEncoding("rot", R, base, 4096)
  pe.prepare(DEV, 128)
  x = r(T, W).to(DT[dtype])
  hdp = -(-(C + R) // 16) * 16
  kv = torch.zeros((8, 2, 1, page, hdp), dtype=DT[dtype], device=DEV)
  bt = torch.zeros((4, 8), dtype=torch.int32, device=DEV)
  bt[2, :4] = torch.tensor([5, 2, 7, 3], dtype=torch.int32)
  dev = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
  rows = None
  for reads, heads, win in ((False, H, window), (True, H + 2, None if window is None else window + 7)):
    m = {"heads": heads, "dim": D, "rot_dim": R, "vdim": Dv, "kv_rank": C, "scale": 0.3, "rot": {"dims": R, "base": base}}
    if win is not None:
      m["mask"] = {"size": win}
    mixer = LatentAttentionMixer("m", W, heads, D, R, Dv, Q, C, 0.3, eps, pe, rotary_interleaved=True, sinks=False, gate_per_head=False, window=win,
                                 keeps_latents=not reads)
    params, P = {}, {}
    for local, ps in mixer.param_specs().items():
      params[local] = torch.zeros(ps.shape, dtype=DT[dtype] if ps.role == "matrix" else torch.float32)
      for piece in ps.sources[0]:
        t = 1 + 0.1 * r(*piece.shape) if len(piece.shape) == 1 else (1.5 * r(*piece.shape) / math.sqrt(piece.shape[-1])).to(DT[dtype])
        params[local][piece.row_start:piece.row_start + piece.shape[0]] = t
        P[piece.file_name] = t.double()
    mixer.bind({k: v.to(DEV) for k, v in params.items()})
    if rows is None:
      rows = plain.latent_rows(x.double(), P, "m.", m, eps)
    want = plain.latent_attention(x.double(), P, "m.", m, eps, rows)
    got = []
    for a, b in ((0, 33), (33, 35), (35, T - 1), (T - 1, T)):
      n = b - a
      lists = {DecodeItems.name: dev([0] if n == 1 else []), PrefillTiles.name: dev([0, 0] if n > 1 else []), PrefillWideTiles.name: dev([0, 0] if n > 1 else [])}
      ctx = SimpleNamespace(dtype=DT[dtype], ws=workspace(), positions=dev(list(range(a, b))), shared={}, work=lists, work_key={DecodeItems.name: (int(n == 1), b)},
                            slot_mapping=[dev([int(bt[2, j // page]) * page + j % page for j in range(a, b)])], block_tables=[bt], num_tokens=n, num_items=1,
                            token_item=dev([0] * n), seq_slot=dev([2]), q_start=dev([0]), q_len=dev([n]), ctx_len=dev([b]))
      got.append(mixer.forward(x[a:b].to(DEV), ctx, LayerCache("paged", 0, kv, not reads, page)).double().cpu())
    assert float((torch.cat(got) - want).abs().max()) <= (1e-4 if dtype == "float32" else 8e-2) * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nh,hd,page,window,ohd", [(3, 48, 16, 24, 40), (7, 96, 64, 70, 80), (9, 128, 64, 64, 112), (16, 256, 64, 100, 192), (2, 272, 16, 33, 264),
                                                   (20, 64, 64, 1, 48)])
def test_keys_on_both_sides_of_a_windows_edge_in_latent_rows(dtype, nh, hd, page, window, ohd):
  """Many query heads on one key/value head whose output is narrower than its rows: the oldest key a token still sees and the
  one before it have scores that no other key comes near."""
  from miniinfer_b200.kernels import ops
  for ctx, new in ((200, 200), (150, 2), (131, 67), (window, 1), (window + 1, 1), (190, 1), (129, 1)):
    p = ctx - 1
    for target in (p - window + 1, p - window):
      if target < 0:
        continue
      qkv, kv, bt, batch = make_attention_case([(ctx, new), (40, 1)], nh, 1, hd, page, DT[dtype], seed=ctx, scale_q=0.01)
      mark = torch.ones(hd) / math.sqrt(hd)
      qkv.view(qkv.shape[0], -1, hd)[:new, :nh] += (30.0 * mark).to(DT[dtype]).to(DEV)
      slot = int(batch.seq_slot[0])
      kv[int(bt[slot, target // page]), 0, 0, target % page] = (6.0 * mark).to(DT[dtype]).to(DEV)
      q = qkv.view(qkv.shape[0], -1, hd)[:new, :nh].double().cpu()
      js = torch.arange(ctx)
      pages = bt[slot].long().cpu()[js // page]
      k, v = kv.cpu()[pages, 0, 0, js % page].double(), kv.cpu()[pages, 1, 0, js % page].double()
      s = torch.einsum("thd,nd->htn", q, k) * 0.25
      w = plain.softmax_over(s, plain.in_window(ctx, window)[ctx - new:][None])
      want = torch.einsum("htn,nd->thd", w, v)[:, :, :ohd].reshape(new, -1)
      # the rows that still look for the marked key must show it, the others must not
      assert float(want.view(new, nh, ohd)[-1].sub(v[target, :ohd]).abs().max()) < 1e-6 if target > p - window else True
      out = torch.zeros((qkv.shape[0], nh * ohd), dtype=DT[dtype], device=DEV)
      ops.attention(out, qkv, kv, bt, batch, nh, 1, hd, 0.25, window, out_hd=ohd)
      assert float((out[:new].double().cpu() - want).abs().max()) <= (3e-5 if dtype == "float32" else 2e-2) * float(want.abs().max()), (ctx, new, target)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,Dv,dims,base,factor", [(4, 2, 24, 40, 16, 300.0, 4.0), (3, 3, 32, 16, 32, 90.0, 1.0), (6, 2, 88, 96, 36, 30000.0, 6.0), (2, 1, 8, 8, 2, 10.0, 0.5)])
def test_normed_heads_rotated_by_divided_frequencies(dtype, H, G, D, Dv, dims, base, factor):
  from miniinfer_b200.kernels import ops
  from miniinfer_b200.parts import LinearScaledRotaryEncoding
  g = torch.Generator().manual_seed(dims + D)
  T, page, eps = 11, 8, 1e-5
  hdp = -(-max(D, Dv) // 16) * 16
  pe = LinearScaledRotaryEncoding("rot", dims, base, 4096, factor=factor)
  pe.prepare(DEV, 64)
  proj = torch.randn((T, H * D + G * (D + Dv)), generator=g).to(DT[dtype])
  qw, kw = 1 + 0.3 * torch.randn((D,), generator=g), 1 + 0.3 * torch.randn((D,), generator=g)
  pos = torch.arange(20, 20 + T)
  p = proj.double()
  q = plain.rotate_pairs(plain.rms(p[:, :H * D].view(T, H, D), eps) * qw.double(), pos, dims, base, factor)
  k = plain.rotate_pairs(plain.rms(p[:, H * D:(H + G) * D].view(T, G, D), eps) * kw.double(), pos, dims, base, factor)
  v = p[:, (H + G) * D:].view(T, G, Dv)
  kv = torch.zeros((6, 2, G, page, hdp), dtype=DT[dtype], device=DEV)
  slots = torch.tensor([3 * page + 5 - j if j < 6 else 4 * page + j for j in range(T)], dtype=torch.int32, device=DEV)
  q_out = torch.full((T, H * hdp), 3.0, dtype=DT[dtype], device=DEV)
  ops.qkv_norm_mix_store(proj.to(DEV), 0, H * D, (H + G) * D, q_out, H, G, D, Dv, eps, True, qw.to(DEV), kw.to(DEV), None, None, 0, slots, kv,
                         rope=pe.rotary_table(), positions=pos.to(torch.int32).to(DEV), interleaved=True)
  qo = q_out.double().cpu().view(T, H, hdp)
  assert float((qo[..., :D] - q).abs().max()) <= tol(dtype) and (hdp == D or float(qo[..., D:].abs().max()) == 0)
  for j in range(T):
    s = int(slots[j])
    assert float((kv[s // page, 0, :, s % page, :D].double().cpu() - k[j]).abs().max()) <= tol(dtype)
    assert float((kv[s // page, 1, :, s % page, :Dv].double().cpu() - v[j]).abs().max()) <= tol(dtype)
