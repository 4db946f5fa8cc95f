"""Plain implementation of the Besolix design: whole sequences, no cache, float64 on the CPU, one function per
mechanism, written from the design's equations and sharing nothing with the package.  It also makes the random
weights of the tests (``make_model``), with distributions under which every mechanism moves the logits.

Notation: ``T`` tokens, ``W`` width, ``H`` query heads, ``G`` key/value heads, ``D`` query/key size, ``R`` rotated
query/key size, ``Dv`` value size, ``Q`` and ``C`` the query and key/value latents, ``K`` taps of a convolution.
"""

from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional, Tuple

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------ small mechanisms


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
  return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def stored_around_zero(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
  """The norm of the residual stream, whose weight is what is added to one."""
  return rms(x, eps) * (1.0 + w)


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float, factor: float = 1.0) -> torch.Tensor:
  """x [T, heads, D]: of a head's first ``dims`` values, 2i and 2i + 1 are rotated together by the angle
  position * base^(-2 i / dims) / factor."""
  f = base ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims) / factor
  a = positions.to(F64)[:, None] * f[None, :]
  cos, sin = a.cos()[:, None, :], a.sin()[:, None, :]
  u, v = x[..., 0:dims:2], x[..., 1:dims:2]
  turned = torch.stack([u * cos - v * sin, v * cos + u * sin], -1).flatten(-2)
  return torch.cat([turned, x[..., dims:]], -1)


def factor_of(m: dict) -> float:
  return float(m["rot"]["scaling"]["factor"]) if m["rot"].get("scaling") else 1.0


def in_window(T: int, size: Optional[int]) -> torch.Tensor:
  """[T, T]: may the row's token see the column's?  Itself and the ``size - 1`` tokens before it."""
  d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
  return (d >= 0) & (d < size) if size else d >= 0


def softmax_over(s: torch.Tensor, seen: torch.Tensor) -> torch.Tensor:
  return torch.softmax(s.masked_fill(~seen, -math.inf), -1)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
  return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
  return z * torch.sigmoid(z)


def short_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
  """x [T, channels], w [channels, K]: token t gets sum_k w[:, K - 1 - k] x[t - k], nothing lying before the start."""
  T, K = x.shape[0], w.shape[1]
  out = torch.zeros_like(x)
  for k in range(K):
    if k < T:
      out[k:] += w[:, K - 1 - k] * x[:T - k]
  return out


def unit(x: torch.Tensor) -> torch.Tensor:
  return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
  """q, k [T, H, D], v [T, H, Dv], g and beta [T, H]; per head the state decays, is corrected towards v along k, is read by q."""
  T, H, D = q.shape
  S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
  out = []
  for t in range(T):
    S = g[t][:, None, None] * S
    u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
    S = S + torch.einsum("hd,hv->hdv", k[t], u)
    out.append(torch.einsum("hdv,hd->hv", S, q[t]))
  return torch.stack(out)


# ------------------------------------------------------------------------------------------ the mixers


def window_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
  T = h.shape[0]
  H, G, D, Dv = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
  rot, factor = m["rot"], factor_of(m)
  pos = torch.arange(T)
  q = rms((h @ W[p + "q"].T).view(T, H, D), eps) * W[p + "q.norm"]
  k = rms((h @ W[p + "k"].T).view(T, G, D), eps) * W[p + "k.norm"]
  q = rotate_pairs(q, pos, int(rot["dims"]), float(rot["base"]), factor)
  k = rotate_pairs(k, pos, int(rot["dims"]), float(rot["base"]), factor).repeat_interleave(H // G, 1)
  v = (h @ W[p + "v"].T).view(T, G, Dv).repeat_interleave(H // G, 1)
  s = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"])
  a = softmax_over(s, in_window(T, m["mask"]["size"] if m.get("mask") else None))
  return torch.einsum("hij,jhd->ihd", a, v).reshape(T, H * Dv) @ W[p + "o"].T


def latent_rows(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
  """What a latent layer keeps of every token: the normed latent [T, C] and the rotated key part [T, R]."""
  C = int(m["kv_rank"])
  kv = h @ W[p + "dkv"].T
  c = rms(kv[:, :C], eps) * W[p + "dkv.norm"]
  return c, rotate_pairs(kv[:, None, C:], torch.arange(h.shape[0]), int(m["rot_dim"]), float(m["rot"]["base"]), factor_of(m))[:, 0]


def latent_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float,
                     rows: Tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
  """``rows``: the latents and rotated key parts, this layer's own or another's."""
  T = h.shape[0]
  H, D, R, Dv = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim"))
  c, k_rot = rows
  q = (rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"] @ W[p + "uq"].T).view(T, H, D + R)
  q_rot = rotate_pairs(q[..., D:], torch.arange(T), R, float(m["rot"]["base"]), factor_of(m))
  k = (c @ W[p + "uk"].T).view(T, H, D)
  v = (c @ W[p + "uv"].T).view(T, H, Dv)
  s = (torch.einsum("ihd,jhd->hij", q[..., :D], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * float(m["scale"])
  a = softmax_over(s, in_window(T, m["mask"]["size"] if m.get("mask") else None))
  o = torch.einsum("hij,jhd->ihd", a, v).reshape(T, H * Dv)
  return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def gated_delta(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
  T = h.shape[0]
  H, G, D, Dv = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
  q, k, v = (silu(short_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v"))
  q = (unit(q.view(T, G, D)) * D ** -0.5).repeat_interleave(H // G, 1)
  k = unit(k.view(T, G, D)).repeat_interleave(H // G, 1)
  beta = torch.sigmoid(h @ W[p + "b"].T)
  g = torch.exp(-torch.exp(W[p + "A_log"]) * torch.nn.functional.softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
  o = delta_rule(q, k, v.view(T, H, Dv), g, beta)
  o = rms(o, eps) * W[p + "norm"] * silu((h @ W[p + "g"].T).view(T, H, Dv))
  return o.reshape(T, H * Dv) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ the model


def feed_forward(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
  return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens, layers_out: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
  """Logits [T, vocab] of one sequence (float32); ``layers_out`` receives the residual stream after every layer."""
  W = {k: v.to(F64) for k, v in W.items()}
  eps = float(cfg["norm"]["eps"])
  x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
  kept = {}
  for i, layer in enumerate(cfg["layers"]):
    p, m = f"l{i}.", layer["mixer"]
    h = stored_around_zero(x, W[p + "norm1"], eps)
    if layer["type"] == "attention":
      y = window_attention(h, W, p + "mix.", m, eps)
    elif layer["type"] == "delta":
      y = gated_delta(h, W, p + "mix.", m, eps)
    elif layer["type"] == "latent_attention":
      src = m.get("kv_from")
      if src is None:
        src = i
        kept[i] = latent_rows(h, W, p + "mix.", m, eps)
      y = latent_attention(h, W, p + "mix.", m, eps, kept[src])
    else:
      raise ValueError(layer["type"])
    x = x + y
    if layer.get("mlp") is not None:
      x = x + feed_forward(stored_around_zero(x, W[p + "norm2"], eps), W, p + "mlp.")
    if layers_out is not None:
      layers_out.append(x.float().clone())
  return (stored_around_zero(x, W["final.norm"], eps) @ W["head"].T).float()


def generate(cfg: dict, W: Dict[str, torch.Tensor], prompt: List[int], n: int) -> List[int]:
  ids = list(prompt)
  for _ in range(n):
    ids.append(int(forward(cfg, W, ids)[-1].argmax()))
  return ids[len(prompt):]


# ------------------------------------------------------------------------------------------ weights for the tests


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
  """Name -> shape of every tensor of a model with this configuration."""
  Wd, V = cfg["width"], cfg["vocab"]
  out: Dict[str, tuple] = {"embed": (V, Wd), "final.norm": (Wd,), "head": (V, Wd)}
  for i, layer in enumerate(cfg["layers"]):
    p, m, q = f"l{i}.", layer["mixer"], f"l{i}.mix."
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    out.update({p + "norm1": (Wd,), q + "o": (Wd, H * Dv)})
    if layer["type"] == "attention":
      G = m["kv_heads"]
      out.update({q + "q": (H * D, Wd), q + "k": (G * D, Wd), q + "v": (G * Dv, Wd), q + "q.norm": (D,), q + "k.norm": (D,)})
    elif layer["type"] == "delta":
      G, K = m["kv_heads"], m["conv"]
      out.update({q + "q": (G * D, Wd), q + "q.conv": (G * D, K), q + "k": (G * D, Wd), q + "k.conv": (G * D, K), q + "v": (H * Dv, Wd),
                  q + "v.conv": (H * Dv, K), q + "b": (H, Wd), q + "a": (H, Wd), q + "A_log": (H,), q + "dt_bias": (H,), q + "norm": (Dv,),
                  q + "g": (H * Dv, Wd)})
    else:
      R, Q, C = m["rot_dim"], m["q_rank"], m["kv_rank"]
      out.update({q + "dq": (Q, Wd), q + "dq.norm": (Q,), q + "uq": (H * (D + R), Q), q + "uk": (H * D, C), q + "uv": (H * Dv, C),
                  q + "g": (H * Dv, Wd)})
      if m.get("kv_from") is None:
        out.update({q + "dkv": (C + R, Wd), q + "dkv.norm": (C,)})
    if layer.get("mlp") is not None:
      F = layer["mlp"]["ff"]
      out.update({p + "norm2": (Wd,), p + "mlp.gate": (F, Wd), p + "mlp.up": (F, Wd), p + "mlp.down": (Wd, F)})
  return out


def make_model(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
  """Random weights, all exactly representable in bfloat16, under which every mechanism moves the logits: projections with
  a fan-in scale (queries and keys larger, so that single keys stand out), norm weights that differ from value to value,
  decays that keep a memory for a few to a hundred tokens, convolutions whose older taps count, gates that open and close."""
  g = torch.Generator().manual_seed(seed)
  W: Dict[str, torch.Tensor] = {}
  for name, shape in tensor_shapes(cfg).items():
    last = name.split(".")[-1]
    r = torch.randn(shape, generator=g)
    if name == "embed":
      t = r
    elif last in ("norm1", "norm2") or name == "final.norm":
      t = 0.3 * r
    elif last == "norm":
      t = 1.0 + 0.3 * r
      if name.endswith("q.norm") or name.endswith("k.norm"):
        t = 1.5 * t
    elif last == "conv":
      t = 0.7 * r
    elif last == "A_log":
      t = r - 0.5
    elif last == "dt_bias":
      t = 1.5 * r - 3.0
    elif last in ("gate", "up", "a", "b", "g"):
      t = r * 2.0 / math.sqrt(shape[-1])
    elif last in ("uq", "uk"):
      t = r * 1.7 / math.sqrt(shape[-1])
    else:
      t = r / math.sqrt(shape[-1])
    W[name] = t.to(torch.bfloat16).float()
  return W


def write_model(cfg: dict, W: Dict[str, torch.Tensor], folder: str, dtype: torch.dtype = torch.bfloat16) -> str:
  from safetensors.torch import save_file
  os.makedirs(folder, exist_ok=True)
  with open(os.path.join(folder, "config.json"), "w") as f:
    json.dump(cfg, f)
  save_file({k: v.to(dtype).contiguous() for k, v in W.items()}, os.path.join(folder, "model.safetensors"))
  return folder


def make_model_dir(cfg: dict, folder: str, seed: int) -> str:
  return write_model(cfg, make_model(cfg, seed), folder)


def read_weights(model_dir: str) -> Dict[str, torch.Tensor]:
  from safetensors.torch import load_file
  return {k: v.float() for k, v in load_file(os.path.join(model_dir, "model.safetensors")).items()}


def read_config(model_dir: str) -> dict:
  with open(os.path.join(model_dir, "config.json"), encoding="utf-8") as f:
    return json.load(f)


# ------------------------------------------------------------------------------------------ configurations


def _mlp(ff):
  return None if ff is None else {"kind": "dense", "ff": ff}


def attention(heads, kv_heads, dim, vdim, window, dims, base, factor, scale, ff) -> dict:
  rot = {"dims": dims, "base": base}
  if factor is not None:
    rot["scaling"] = {"factor": factor}
  m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": scale}
  if window is not None:
    m["mask"] = {"size": window}
  return {"type": "attention", "mlp": _mlp(ff), "mixer": m}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, base, scale, ff, kv_from=None) -> dict:
  m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
       "rot": {"dims": rot_dim, "base": base}}
  if window is not None:
    m["mask"] = {"size": window}
  if kv_from is not None:
    m["kv_from"] = kv_from
  return {"type": "latent_attention", "mlp": _mlp(ff), "mixer": m}


def delta(heads, kv_heads, dim, vdim, conv, ff) -> dict:
  return {"type": "delta", "mlp": _mlp(ff), "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def model(vocab, width, eps, *layers) -> dict:
  return {"architecture": "Besolix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": list(layers)}


# Configurations that differ in every size, in the order of their layers and in what is there at all.  A: windows of 24 and 20
# tokens on pages of 16, a reader of layer 0's latents with more heads and twice the window, one key/value head for four query
# heads, values larger than keys, a layer without a feed-forward.  B: the delta rule first, a convolution of one tap, as many
# key/value heads as query heads, values smaller than keys, a window of one token, no scaling, a latent layer of one head whose
# readers see every earlier token and three tokens, whole heads rotated.  C: heads of 64 and 128 with windows of 96 and 150 (the
# tensor-core and tensor-copy kernels on pages of 64), a delta rule of 128 x 64, a latent of 96 + 32.  D: odd sizes - a width of
# 72, a vocabulary of 333, sixteen query heads on one key/value head, a delta rule of 40 x 8 behind two taps, latent rows of
# more than 256 values, an eps of 1e-3, a reader that stands behind another latent layer.  E: three latent layers in a row over
# one cache - nine heads, windows of 200, 64 and 130 -, a delta rule of 48 x 80 with six heads on two behind six taps.
# F: no size is a multiple of 8, and few are even.
CONFIGS = {
  "A": model(300, 64, 1e-5,
             latent(3, 24, 8, 16, 24, 40, 24, 10000.0, 0.2, 40),
             attention(4, 1, 24, 40, 20, 16, 5000.0, 4.0, 0.25, 48),
             delta(4, 2, 16, 24, 4, 40),
             latent(5, 16, 8, 24, 32, 40, 50, 10000.0, 0.25, None, kv_from=0),
             delta(4, 2, 16, 24, 4, None),
             attention(4, 1, 24, 40, 20, 16, 5000.0, 4.0, 0.25, 24)),
  "B": model(200, 32, 1e-6,
             delta(2, 2, 32, 16, 1, 24),
             latent(1, 16, 16, 32, 8, 16, 9, 500.0, 0.25, None),
             attention(2, 2, 16, 8, 1, 16, 100.0, None, 0.25, 16),
             latent(2, 8, 16, 8, 16, 16, None, 500.0, 0.25, 16, kv_from=1),
             attention(6, 3, 32, 16, 7, 32, 800.0, 2.5, 0.2, None),
             latent(1, 16, 16, 32, 8, 16, 3, 500.0, 0.25, 24, kv_from=1)),
  "C": model(500, 128, 1e-6,
             attention(8, 2, 64, 64, 96, 32, 20000.0, 3.0, 0.125, 96),
             latent(4, 32, 32, 32, 48, 96, 100, 8000.0, 0.125, 64),
             delta(4, 1, 128, 64, 4, 64),
             attention(4, 2, 128, 128, 150, 128, 50000.0, 16.0, 0.09, None),
             latent(4, 64, 32, 16, 64, 96, 70, 8000.0, 0.1, 96, kv_from=1)),
  "D": model(333, 72, 1e-3,
             latent(2, 40, 8, 24, 56, 264, 33, 3000.0, 0.15, 24),
             latent(3, 8, 16, 8, 24, 32, 17, 700.0, 0.2, 40),
             attention(16, 1, 32, 48, 33, 8, 300.0, 1.5, 0.2, 24),
             delta(6, 3, 40, 8, 2, None),
             latent(1, 16, 8, 40, 16, 264, 40, 3000.0, 0.2, 24, kv_from=0),
             attention(5, 5, 8, 8, 40, 4, 60.0, 7.0, 0.4, None)),
  "E": model(400, 96, 1e-5,
             latent(9, 32, 16, 24, 40, 112, 200, 8000.0, 0.15, 64),
             latent(9, 16, 16, 24, 24, 112, 64, 8000.0, 0.2, None, kv_from=0),
             latent(2, 32, 16, 48, 40, 112, 130, 8000.0, 0.15, 32, kv_from=0),
             delta(6, 2, 48, 80, 6, 64)),
  "F": model(101, 37, 1e-4,
             latent(3, 9, 6, 5, 11, 21, 13, 400.0, 0.3, 27),
             delta(3, 3, 7, 9, 3, 18),
             attention(3, 1, 11, 7, 10, 6, 60.0, 3.0, 0.3, None),
             latent(1, 5, 6, 13, 7, 21, 6, 400.0, 0.35, 35, kv_from=0),
             delta(5, 1, 10, 3, 2, None)),
}


def peaky_model():
  """(configuration, weights) under which single keys stand out: windows of 100 and of 70 tokens - 130 for a reader of the first
  layer's latents -, scores spread over tens of units by large scales."""
  cfg = model(200, 64, 1e-5,
              latent(2, 32, 16, 32, 32, 48, 100, 10000.0, 0.35, None),
              attention(2, 1, 32, 48, 70, 24, 9000.0, 2.0, 1.0, 48),
              latent(3, 16, 16, 24, 40, 48, 130, 10000.0, 0.5, None, kv_from=0),
              delta(2, 1, 32, 32, 3, 32))
  return cfg, make_model(cfg, 77)
