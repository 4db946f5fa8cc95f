"""Token embedding and LM head.

Embedding: a row lookup (miniinfer/layers/embedding.py:23-27), written as float32 because it starts
the residual stream.  LM head: ``x @ W^T`` (embedding.py:29-32) with float32 logits; it uses the
embedding's table when the configuration ties them.  The reference decides tying by whether the
file has ``lm_head.weight`` (embedding.py:41-48); here ``tie_word_embeddings`` decides and the file
is checked against it.
"""

from __future__ import annotations

from typing import Dict, Optional

import torch

from ..kernels import ops
from .base import Embedding, Head, ParamSpec, whole


class TokenEmbedding(Embedding):
  """``scale``: a constant the looked-up row is multiplied with (1: none).  ``tensor``: the table's name in the weights
  file (default ``<name>.weight``).  ``copies``: the row is written that many times side by side, for models whose
  residual stream is several streams that start equal."""

  def __init__(self, name: str, vocab_size: int, hidden_size: int, scale: float = 1.0, tensor: Optional[str] = None, copies: int = 1):
    super().__init__(name)
    if copies < 1:
      raise ValueError(f"{name}: copies must be positive, got {copies}")
    self.vocab_size = vocab_size
    self.hidden_size = hidden_size
    self.scale = float(scale)
    self.tensor = tensor or f"{name}.weight"
    self.copies = copies

  def param_specs(self) -> Dict[str, ParamSpec]:
    shape = (self.vocab_size, self.hidden_size)
    return {"weight": ParamSpec(shape, "table", [whole(self.tensor, shape)])}

  def forward(self, ids: torch.Tensor, ctx) -> torch.Tensor:
    out = ctx.ws.buffer("resid", (ids.shape[0], self.copies * self.hidden_size), torch.float32)
    if self.copies != 1:
      ops.embedding(out, self.weight, ids, self.scale, self.copies)
    elif self.scale == 1.0:
      ops.embedding(out, self.weight, ids)
    else:
      ops.embedding(out, self.weight, ids, self.scale)
    return out


class LMHead(Head):
  """``softcap`` > 0: the logits leave as ``softcap * tanh(logits / softcap)``."""

  def __init__(self, name: str, vocab_size: int, hidden_size: int, tied_to: Optional[TokenEmbedding] = None,
               tensor: Optional[str] = None, softcap: float = 0.0):
    super().__init__(name)
    if not softcap >= 0:
      raise ValueError(f"{name}: softcap must not be negative, got {softcap!r}")
    self.vocab_size = vocab_size
    self.hidden_size = hidden_size
    self.tied_to = tied_to
    self.softcap = float(softcap)
    self.tensor = tensor or f"{name}.weight"

  def param_specs(self) -> Dict[str, ParamSpec]:
    if self.tied_to is not None:
      return {}
    shape = (self.vocab_size, self.hidden_size)
    return {"weight": ParamSpec(shape, "matrix", [whole(self.tensor, shape)])}

  def table(self) -> torch.Tensor:
    return self.tied_to.weight if self.tied_to is not None else self.weight

  def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
    out = ctx.ws.buffer("logits", (x.shape[0], self.vocab_size), torch.float32)
    ops.linear(out, x, self.table())
    if self.softcap > 0:
      ops.softcap(out, self.softcap)
    return out
