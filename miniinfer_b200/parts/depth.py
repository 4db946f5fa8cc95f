"""Pre-norm layers whose results are averaged over depth.

With ``X_0`` the rows the embedding left and ``X_(i+1)`` the result of layer ``i``, which is

    ``X_(i+1) = x + mult * f1 + mult * f2``,   ``f1 = mixer(norm1(x))``, ``f2 = ff(norm2(x + mult * f1))``,

what the layer hands on is ``x' = sum_(j = 0 .. i+1) w[j] X_j`` with ``i + 2`` learned weights of its own.  ``mult`` is a constant.

The first addition of a layer and the norm behind it are one kernel, and so are the second, the average and the next
layer's norm (``ops.residual_step``): a layer leaves its last sublayer's output pending (``PendingAverage``) for whoever reads
the stream next - the next layer or the final ``DepthAverageNorm``.  The stream and everything that is kept of earlier
layers are float32 whatever the compute dtype, and live in the step's workspace: the embedding's rows stay where they are,
the stream has a buffer of its own, and the results of the layers lie behind one another in a third.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from ..kernels import ops
from .base import Block, FeedForward, Mixer, Norm, ParamSpec, Part, whole


@dataclass
class PendingAverage:
  """A layer's last output ``y`` that is not yet in the stream ``x``, the average the layer ends in (``weights`` over ``first``,
  ``n_later`` rows of ``later`` and the layer's result) and where its result is kept for later layers (None: nobody asks)."""

  x: torch.Tensor
  y: Optional[torch.Tensor]
  mult: float
  weights: torch.Tensor
  first: torch.Tensor
  later: Optional[torch.Tensor]
  n_later: int
  keep: Optional[torch.Tensor]

  def settle(self, norm: Norm, ctx, x_out: Optional[torch.Tensor], rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The normed rows of the averaged stream; ``x_out`` receives the stream itself."""
    return _step(norm, ctx, self.x, self.y, self.mult, x_out, rows, weights=self.weights, first=self.first, later=self.later,
                 n_later=self.n_later, keep=self.keep)


def _step(norm: Norm, ctx, x, y, mult, x_out, rows=None, **average) -> torch.Tensor:
  form = norm.as_row_norm()
  if form is not None:
    R = x.shape[0] if rows is None else rows.shape[0]
    out = ctx.ws.buffer("normed" if rows is None else "normed_rows", (R, x.shape[1]), ctx.dtype)
    ops.residual_step(out, x, y, mult, x_out, form, rows, **average)
    return out
  # a norm of another kind: the stream first, then the norm's own kernel
  if x_out is None:
    x_out = ctx.ws.buffer("depth_last", tuple(x.shape), torch.float32)
  ops.residual_step(None, x, y, mult, x_out, None, None, **average)
  return norm.add_norm(x_out, None, ctx) if rows is None else norm.norm_rows(x_out, None, rows, ctx)


class DepthAverageBlock(Block):
  """Layer number ``index`` of ``depth``: a mixer behind ``mixer_norm`` and, if there is one, a feed-forward behind
  ``ffn_norm``.  File tensor of the weights: ``<name>.dwa`` (``weights_name``), ``index + 2`` numbers."""

  def __init__(self, name: str, index: int, depth: int, width: int, mixer_norm: Norm, mixer: Mixer, ffn_norm: Optional[Norm],
               ffn: Optional[FeedForward], mult: float = 1.0, weights_name: Optional[str] = None):
    super().__init__(name)
    if not (0 <= index < depth):
      raise ValueError(f"{name}: index={index} must lie in 0..{depth - 1}")
    if ffn is not None and ffn_norm is None:
      raise ValueError(f"{name}: a feed-forward needs its norm")
    self.index, self.depth, self.width = index, depth, width
    self.mixer_norm, self.mixer = mixer_norm, mixer
    self.ffn = ffn
    self.ffn_norm = ffn_norm if ffn is not None else None
    self.mult = float(mult)
    self.weights_name = weights_name or f"{name}.dwa"

  def sub_parts(self) -> List[Part]:
    return [self.mixer_norm, self.mixer] + ([self.ffn_norm, self.ffn] if self.ffn is not None else [])

  def mixer_part(self) -> Optional[Mixer]:
    return self.mixer

  def param_specs(self):
    n = self.index + 2
    return {"weights": ParamSpec((n,), "vector", [whole(self.weights_name, (n,))], init="mean_noise")}

  def forward(self, resid: torch.Tensor, pending, ctx, cache):
    T = resid.shape[0]
    stream = ctx.ws.buffer("depth_stream", (T, self.width), torch.float32)
    if self.index == 0:
      if pending is not None:
        raise RuntimeError(f"{self.name}: the first layer of a depth average starts from the embedding's rows alone")
      x = resid                                  # X_0 stays as it is; the stream moves to its own buffer with the first addition
      h = _step(self.mixer_norm, ctx, x, None, self.mult, None)
    else:
      if not isinstance(pending, PendingAverage):
        raise TypeError(f"{self.name}: a layer of a depth average continues the layer before it")
      x = stream
      h = pending.settle(self.mixer_norm, ctx, stream)
    y = self.mixer.forward(h, ctx, cache)
    if self.ffn is not None:
      h = _step(self.ffn_norm, ctx, x, y, self.mult, stream)
      x, y = stream, self.ffn.forward(h, ctx)
    # the results of the layers 0 .. index - 1 are kept; this layer's own is, unless it is the last
    later = ctx.ws.buffer("depth_results", (self.depth - 1, T, self.width), torch.float32) if self.depth > 1 else None
    keep = later[self.index] if self.index + 1 < self.depth else None
    return PendingAverage(x, y, self.mult, self.weights, resid, later, self.index, keep)


class DepthAverageNorm(Norm):
  """The norm behind the last layer of a depth average: the last average and ``norm`` in one kernel, for the wanted rows."""

  def __init__(self, name: str, norm: Norm):
    super().__init__(name)
    self.norm = norm

  def sub_parts(self) -> List[Part]:
    return [self.norm]

  def add_norm(self, resid: torch.Tensor, delta, ctx) -> torch.Tensor:
    if not isinstance(delta, PendingAverage):
      return self.norm.add_norm(resid, delta, ctx)
    return delta.settle(self.norm, ctx, None)

  def norm_rows(self, resid: torch.Tensor, delta, rows: torch.Tensor, ctx) -> torch.Tensor:
    if not isinstance(delta, PendingAverage):
      return self.norm.norm_rows(resid, delta, rows, ctx)
    return delta.settle(self.norm, ctx, None, rows)
