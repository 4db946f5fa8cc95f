"""What a layer asks of the cache manager.

The reference has one uniform store for all layers (``MHAKVCacheStorage``,
miniinfer/kvcache/memory_pool.py:18-64).  Here every layer states its need as data; layers with the
same need form a group that has pages (or state slots) of its own.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple, Union


@dataclass(frozen=True)
class PagedKVSpec:
  """Keys and values of every position (``window is None``) or of the last ``window`` positions; with
  ``keep_first`` the first positions of a request stay as well, whatever the window has passed.  With ``chunk`` (and no
  window) those of the chunk of that many positions, counted from position 0, which the next position lies in."""

  num_kv_heads: int
  head_dim: int
  window: Optional[int] = None
  keep_first: int = 0
  chunk: Optional[int] = None

  def __post_init__(self):
    if self.num_kv_heads <= 0 or self.head_dim <= 0:
      raise ValueError("num_kv_heads and head_dim must be positive")
    if self.window is not None and self.window <= 0:
      raise ValueError("window must be positive or None")
    if self.keep_first < 0:
      raise ValueError("keep_first must not be negative")
    if self.chunk is not None and (self.chunk <= 0 or self.window is not None):
      raise ValueError("chunk must be positive or None, and goes without a window")

  @property
  def reach(self) -> Optional[int]:
    """The most positions a query looks back on (its own included), or None: all of them."""
    return self.window if self.window is not None else self.chunk

  def first_needed(self, length: int) -> int:
    """The first position, kept first ones aside, that a query at position ``length`` (the next one) or later can see."""
    if self.window is not None:
      return max(0, length - self.window + 1)
    return length // self.chunk * self.chunk if self.chunk is not None else 0


@dataclass(frozen=True)
class FixedStateSpec:
  """A tensor of fixed shape for each live request, zero when the request is admitted."""

  shape: Tuple[int, ...]
  dtype: str = "float32"

  def __post_init__(self):
    if any(int(s) <= 0 for s in self.shape):
      raise ValueError("state shape must be positive")


@dataclass(frozen=True)
class CompositeSpec:
  """What a mixer made of several mixers keeps: the needs of its members, in their order.  The layer's cache is then
  handed over as one ``LayerCache`` per member (``LayerCache.members``)."""

  members: Tuple[Union[PagedKVSpec, FixedStateSpec], ...]

  def __post_init__(self):
    if not self.members:
      raise ValueError("a composite cache need has at least one member")


CacheSpec = Union[PagedKVSpec, FixedStateSpec, CompositeSpec]


def shared_need(specs) -> CacheSpec:
  """The need of one cache that several layers read: keys and values of one shape for as long as any of them can see them -
  the widest window, or everything once a reader sees every earlier key or the readers mix windows and chunks.
  ``ValueError`` if the layers differ in what a row holds."""
  first = specs[0]
  if all(s == first for s in specs):
    return first
  if not all(isinstance(s, PagedKVSpec) and (s.num_kv_heads, s.head_dim) == (first.num_kv_heads, first.head_dim) for s in specs):
    raise ValueError("layers that share a cache differ in what they keep in it")
  windows = [s.window for s in specs]
  if all(w is not None for w in windows):
    return PagedKVSpec(first.num_kv_heads, first.head_dim, max(windows), max(s.keep_first for s in specs))
  return PagedKVSpec(first.num_kv_heads, first.head_dim)


def flatten_specs(layer_specs):
  """The needs of all layers, the members of composite ones one by one, without the layers that keep nothing."""
  out = []
  for spec in layer_specs:
    if isinstance(spec, CompositeSpec):
      out.extend(spec.members)
    elif spec is not None:
      out.append(spec)
  return out
