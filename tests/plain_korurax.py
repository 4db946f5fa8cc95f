"""Plain implementation of the Korurax design: whole sequences, no cache, float64 on the CPU, one function per
mechanism, written from the design's equations and sharing nothing with the package.  It also makes the random
weights of the tests (``make_model``), with distributions under which every mechanism moves the logits.

Notation: ``T`` tokens, ``W`` width, ``H`` query heads, ``G`` key/value heads, ``D`` query/key size, ``R`` rotated
query/key size, ``Dv`` value size, ``Q`` and ``C`` the query and key/value latents, ``E`` experts.
"""

from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------ small mechanisms


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
  """A weight, no bias; the variance is the mean of the squared deviations."""
  d = x - x.mean(-1, keepdim=True)
  return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
  return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def depth_average(history: List[torch.Tensor], w: torch.Tensor) -> torch.Tensor:
  """history: the embedding rows and every layer's result so far; a weight each."""
  out = torch.zeros_like(history[0])
  for j, X in enumerate(history):
    out = out + w[j] * X
  return out


def rotate_half(x: torch.Tensor, positions: torch.Tensor, base: float) -> torch.Tensor:
  """x [T, heads, R]: value i of a head is rotated with value i + R / 2 by the angle position * base^(-2 i / R)."""
  R = x.shape[-1]
  f = base ** (-2.0 * torch.arange(R // 2, dtype=F64) / R)
  a = positions.to(F64)[:, None] * f[None, :]
  cos, sin = a.cos()[:, None, :], a.sin()[:, None, :]
  u, v = x[..., :R // 2], x[..., R // 2:]
  return torch.cat([u * cos - v * sin, v * cos + u * sin], -1)


def same_chunk(T: int, size: Optional[int]) -> torch.Tensor:
  """[T, T]: may the row's token see the column's?  Earlier tokens (and itself) of its own chunk of ``size`` positions."""
  i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
  seen = j <= i
  return seen if not size else seen & (i // size == j // size)


def distance_bias(T: int, r1: torch.Tensor, r2: torch.Tensor) -> torch.Tensor:
  """[H, T, T]: what is taken off the score of a query and a key that far behind it."""
  d = (torch.arange(T, dtype=F64)[:, None] - torch.arange(T, dtype=F64)[None, :]).clamp(min=0)
  return r1[:, None, None] * torch.log(1.0 + r2[:, None, None] * d)


def softmax_with_sink(s: torch.Tensor, seen: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
  """s [H, T, T] over the last axis; ``sink [H]``: a logit that joins the denominator alone."""
  s = s.masked_fill(~seen, -math.inf)
  if sink is None:
    return torch.softmax(s, -1)
  extra = sink[:, None, None].expand(s.shape[0], s.shape[1], 1)
  return torch.softmax(torch.cat([s, extra], -1), -1)[..., :-1]


# ------------------------------------------------------------------------------------------ the mixers


def chunked_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict) -> torch.Tensor:
  T = h.shape[0]
  H, G, D, Dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
  q = (h @ W[p + "q"].T).view(T, H, D)
  k = (h @ W[p + "k"].T).view(T, G, D).repeat_interleave(H // G, 1)
  v = (h @ W[p + "v"].T).view(T, G, Dv).repeat_interleave(H // G, 1)
  s = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"]) - distance_bias(T, W[p + "r1"], W[p + "r2"])
  size = m["mask"]["size"] if m.get("mask") else None
  a = softmax_with_sink(s, same_chunk(T, size), W[p + "sink"])
  o = torch.einsum("hij,jhd->ihd", a, v) * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
  return o.reshape(T, H * Dv) @ W[p + "o"].T


def latent_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
  T = h.shape[0]
  H, D, R, Dv, C = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
  pos = torch.arange(T)
  q = (rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).view(T, H, D + R)
  kv = h @ W[p + "dkv"].T
  c = rms_norm(kv[:, :C], W[p + "dkv.norm"], eps)
  k_rot = rotate_half(kv[:, None, C:], pos, float(m["rot"]["base"]))[:, 0]
  q_rot = rotate_half(q[..., D:], pos, float(m["rot"]["base"]))
  k = (c @ W[p + "uk"].T).view(T, H, D)
  v = (c @ W[p + "uv"].T).view(T, H, Dv)
  s = (torch.einsum("ihd,jhd->hij", q[..., :D], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * float(m["scale"])
  a = softmax_with_sink(s, same_chunk(T, None), None)
  return torch.einsum("hij,jhd->ihd", a, v).reshape(T, H * Dv) @ W[p + "o"].T


def mixer(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, layer: dict, eps: float) -> torch.Tensor:
  if layer["type"] == "attention":
    return chunked_attention(h, W, p, layer["mixer"])
  if layer["type"] == "latent_attention":
    return latent_attention(h, W, p, layer["mixer"], eps)
  raise ValueError(layer["type"])


# ------------------------------------------------------------------------------------------ the feed-forwards


def clamped_glu(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, limit: float) -> torch.Tensor:
  g = torch.clamp(h @ W[p + "gate"].T, max=limit)
  u = torch.clamp(h @ W[p + "up"].T, -limit, limit)
  return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def mixture(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, mlp: dict) -> torch.Tensor:
  E, top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
  s = torch.sigmoid(h @ W[p + "router"].T)
  chosen = torch.topk(s, top, dim=-1)
  weights = chosen.values / (chosen.values.sum(-1, keepdim=True) + 1e-20) * float(mlp["router"]["scale"])
  out = torch.zeros_like(h)
  for e in range(E):
    y = torch.relu(h @ W[f"{p}e{e}.up"].T) ** 2 @ W[f"{p}e{e}.down"].T
    out = out + (weights * (chosen.indices == e)).sum(-1, keepdim=True) * y
  return out


def feed_forward(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, mlp: dict) -> torch.Tensor:
  return clamped_glu(h, W, p, float(mlp["limit"])) if mlp["kind"] == "dense" else mixture(h, W, p, mlp)


# ------------------------------------------------------------------------------------------ the model


def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens, layers_out: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
  """Logits [T, vocab] of one sequence (float32); ``layers_out`` receives what every layer hands on."""
  W = {k: v.to(F64) for k, v in W.items()}
  eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
  x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
  history = [x]
  for i, layer in enumerate(cfg["layers"]):
    p = f"l{i}."
    x = x + m * mixer(layer_norm(x, W[p + "norm1"], eps), W, p + "mix.", layer, eps)
    if layer.get("mlp") is not None:
      x = x + m * feed_forward(layer_norm(x, W[p + "norm2"], eps), W, p + "mlp.", layer["mlp"])
    history.append(x)
    x = depth_average(history, W[p + "dwa"])
    if layers_out is not None:
      layers_out.append(x.float().clone())
  cap = float(cfg["logit_softcap"])
  return (cap * torch.tanh(layer_norm(x, W["final.norm"], eps) @ W["embed"].T / cap)).float()


def generate(cfg: dict, W: Dict[str, torch.Tensor], prompt: List[int], n: int) -> List[int]:
  ids = list(prompt)
  for _ in range(n):
    ids.append(int(forward(cfg, W, ids)[-1].argmax()))
  return ids[len(prompt):]


# ------------------------------------------------------------------------------------------ weights for the tests


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
  """Name -> shape of every tensor of a model with this configuration."""
  Wd, V = cfg["width"], cfg["vocab"]
  out: Dict[str, tuple] = {"embed": (V, Wd), "final.norm": (Wd,)}
  for i, layer in enumerate(cfg["layers"]):
    p, m, q = f"l{i}.", layer["mixer"], f"l{i}.mix."
    out.update({p + "norm1": (Wd,), p + "dwa": (i + 2,)})
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    if layer["type"] == "attention":
      G = m["kv_heads"]
      out.update({q + "q": (H * D, Wd), q + "k": (G * D, Wd), q + "v": (G * Dv, Wd), q + "r1": (H,), q + "r2": (H,),
                  q + "sink": (H,), q + "g": (H, Wd), q + "o": (Wd, H * Dv)})
    else:
      R, Q, C = m["rot_dim"], m["q_rank"], m["kv_rank"]
      out.update({q + "dq": (Q, Wd), q + "dq.norm": (Q,), q + "uq": (H * (D + R), Q), q + "dkv": (C + R, Wd), q + "dkv.norm": (C,),
                  q + "uk": (H * D, C), q + "uv": (H * Dv, C), q + "o": (Wd, H * Dv)})
    mlp = layer.get("mlp")
    if mlp is not None:
      q = p + "mlp."
      out[p + "norm2"] = (Wd,)
      if mlp["kind"] == "dense":
        F = mlp["ff"]
        out.update({q + "gate": (F, Wd), q + "up": (F, Wd), q + "down": (Wd, F)})
      else:
        F = mlp["expert"]["ff"]
        out[q + "router"] = (mlp["router"]["experts"], Wd)
        for e in range(mlp["router"]["experts"]):
          out.update({f"{q}e{e}.up": (F, Wd), f"{q}e{e}.down": (Wd, F)})
  return out


def make_model(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
  """Random weights, all exactly representable in bfloat16, under which every mechanism moves the logits: projections with
  a fan-in scale (queries and keys larger, so that single keys stand out; gate and up rows larger, so that the clamps
  bite), norm weights around one, distance biases between nothing and a few units over a hundred tokens, sinks of the
  size of a good score, depth weights in which every earlier layer counts, routers whose scores stand apart."""
  g = torch.Generator().manual_seed(seed)
  W: Dict[str, torch.Tensor] = {}
  for name, shape in tensor_shapes(cfg).items():
    last = name.split(".")[-1]
    r = torch.randn(shape, generator=g)
    if name == "embed":
      t = r
    elif last in ("norm1", "norm2", "norm"):
      t = 1.0 + 0.3 * r
    elif last == "dwa":
      t = 0.5 * r / math.sqrt(shape[0])
      t[-1] += 0.8
    elif last == "r1":
      t = 0.2 + 0.8 * torch.rand(shape, generator=g)
    elif last == "r2":
      t = torch.exp(-1.5 + r)
    elif last == "sink":
      t = 1.5 + r
    elif last == "router":
      t = r * 2.5 / math.sqrt(shape[-1])
    elif last in ("gate", "up"):
      t = r * 2.0 / math.sqrt(shape[-1])
    elif last in ("q", "k", "uq", "uk"):
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


def dense(ff, limit) -> dict:
  return {"kind": "dense", "ff": ff, "limit": limit}


def moe(ff, experts, top, scale) -> dict:
  return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def attention(heads, kv_heads, dim, vdim, chunk, scale, mlp) -> dict:
  return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                                     "mask": {"size": chunk}, "scale": scale}}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, base, scale, mlp) -> dict:
  return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
                                                            "kv_rank": kv_rank, "scale": scale, "rot": {"dims": rot_dim, "base": base}}}


def model(vocab, width, eps, mult, cap, *layers) -> dict:
  return {"architecture": "Korurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "logit_softcap": cap,
          "layers": list(layers)}


# Configurations that differ in every size, in the order of their layers and in what is there at all.  A: chunks of 24
# tokens on pages of 16, one key/value head for four query heads, sizes that are no multiple of 16, values larger than keys, a
# chunked layer with a dense feed-forward, a latent layer with a mixture, a layer without a feed-forward.  B: as many
# key/value heads as query heads, chunks of 7 tokens beside chunks of 64, values smaller than keys, one head in a latent
# layer, a router that takes all of its experts and one that takes one, multipliers of 1.  C: heads of 64 and chunks of 96
# (the tensor-core and tensor-copy kernels on pages of 64), a latent of 128.  D: odd sizes - a width of 72, a vocabulary of
# 333, sixteen query heads on one key/value head (and gates that make no multiple of 8 columns), chunks of 33, 40 experts of
# which a token takes 6, a multiplier above 1, an eps of 1e-3, a cap of 4 that bites, latent rows of more than 256 values.
# E: two chunk sizes on heads of 128 and 64 (three query heads a key/value head), chunks larger than a tile.
CONFIGS = {
  "A": model(300, 64, 1e-5, 0.5, 20.0,
             attention(4, 1, 24, 40, 24, 0.3, dense(40, 1.5)),
             latent(3, 24, 8, 16, 24, 40, 10000.0, 0.2, moe(24, 5, 2, 2.5)),
             attention(4, 1, 24, 40, 24, 0.3, None),
             latent(3, 24, 8, 16, 24, 40, 10000.0, 0.2, dense(40, 0.7)),
             attention(2, 2, 16, 16, 50, 0.4, moe(16, 4, 3, 0.8))),
  "B": model(200, 32, 1e-6, 1.0, 50.0,
             latent(1, 16, 16, 32, 8, 16, 500.0, 0.25, moe(16, 3, 3, 1.0)),
             attention(2, 2, 16, 8, 7, 0.25, moe(24, 4, 1, 1.7)),
             attention(6, 3, 32, 16, 64, 0.2, None)),
  "C": model(500, 128, 1e-6, 0.8, 30.0,
             attention(8, 2, 64, 64, 96, 0.125, moe(64, 8, 3, 1.5)),
             latent(4, 32, 32, 32, 48, 96, 20000.0, 0.125, dense(96, 1.2)),
             attention(8, 2, 64, 64, 96, 0.125, dense(64, 2.0)),
             latent(4, 32, 32, 32, 48, 96, 20000.0, 0.125, moe(64, 8, 3, 1.5))),
  "D": model(333, 72, 1e-3, 1.3, 4.0,
             latent(2, 40, 8, 24, 56, 264, 3000.0, 0.3, moe(16, 40, 6, 3.0)),
             attention(16, 1, 32, 48, 33, 0.3, dense(24, 1.0)),
             attention(5, 5, 8, 8, 40, 0.5, moe(16, 40, 6, 0.5))),
  "E": model(400, 96, 1e-5, 0.9, 25.0,
             attention(4, 2, 128, 128, 200, 0.1, dense(64, 1.0)),
             attention(6, 2, 64, 64, 130, 0.15, moe(32, 6, 2, 1.2)),
             latent(9, 32, 16, 24, 40, 112, 8000.0, 0.2, None)),
}


def peaky_model():
  """(configuration, weights) under which single keys stand out: chunks of 100 and of 70 tokens, scores spread over tens of
  units by large scales, distance biases of next to nothing over a chunk, sinks near the largest scores."""
  cfg = model(200, 64, 1e-5, 0.9, 30.0,
              attention(4, 2, 64, 64, 100, 0.45, None),
              latent(2, 32, 16, 32, 32, 48, 10000.0, 0.4, dense(48, 2.0)),
              attention(2, 1, 32, 48, 70, 0.6, moe(16, 4, 2, 1.0)))
  W = make_model(cfg, 77)
  for p in ("l0.mix.", "l2.mix."):
    W[p + "r1"] = (0.3 * W[p + "r1"]).to(torch.bfloat16).float()
    W[p + "sink"] = W[p + "sink"] + 6.0
  return cfg, W
