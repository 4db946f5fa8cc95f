"""Besolix, put together from parts.

Per layer a pre-norm layer (``PreNormBlock``; RMS norms with a weight stored around zero).  The mixer is one of

  * ``latent_attention`` - windowed attention through a latent with a rotated key part shared by all heads and a gate a value
    (``LatentAttentionMixer`` with those options).  A layer with ``kv_from: j`` has no down-projection of its own to keys and
    values: its run-list entry reads the cache that layer ``j`` writes;
  * ``attention`` - windowed grouped-query attention with normed, interleaved-rotated heads (``GatedAttentionMixer`` with those
    options), the frequencies divided by a constant (``LinearScaledRotaryEncoding``);
  * ``delta`` - a gated delta rule behind short convolutions, with one decay a head and a SiLU gate, each from a projection of
    its own (``GatedDeltaMixer`` with those options).

The feed-forward is dense, ``W_down (gelu_tanh(W_gate h) * W_up h)``, or absent.  Around the layers: an embedding, a final norm
(stored around zero as well) and an untied head.  Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``,
``l<i>.mlp.{gate,up,down}``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.model_config import BesolixConfig
from ..config.registry import register_model
from ..parts import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, LMHead, TokenEmbedding, make
from .spec import LayerRun, ModelSpec


@register_model("Besolix", BesolixConfig)
def build_besolix(cfg: BesolixConfig) -> ModelSpec:
  W, eps = cfg.width, cfg.norm_eps
  embedding = TokenEmbedding("embed", cfg.vocab, W, tensor="embed")
  blocks, encodings, unused, run_list = [], {}, [], []

  def rotary(rot):
    factor = rot.scaling["factor"] if rot.scaling is not None else 1.0
    key = (rot.dims, rot.base, factor)
    if key not in encodings:      # layers that rotate alike share a table
      encodings[key] = make(POSITION_ENCODINGS, "linear_scaled_rotary", f"rot{len(encodings)}", rot.dims, rot.base,
                            cfg.max_position_embeddings, factor=factor)
    return encodings[key]

  def norm(name):
    return make(NORMS, "rmsnorm", name, W, eps, offset=1.0, weight_name=name)

  for i in range(len(cfg.layers)):
    p = f"l{i}"
    kind, m, ff = cfg.type_of(i), cfg.mixer_of(i), cfg.ff_of(i)
    cache_of = None
    if kind == "latent_attention":
      cache_of = m.kv_from
      mixer = make(MIXERS, "latent_attention", f"{p}.mix", W, m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, eps,
                   rotary(m.rot), rotary_interleaved=True, sinks=False, gated=True, gate_per_head=False, window=m.window,
                   keeps_latents=cache_of is None)
    elif kind == "attention":
      mixer = make(MIXERS, "gated_attention", f"{p}.mix", W, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, eps, m.window, sinks=False,
                   gated=False, rotary=rotary(m.rot), rotary_interleaved=True, norm_weights=True)
    else:
      mixer = make(MIXERS, "gated_delta", f"{p}.mix", W, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, None, None, eps, gate="silu")
    ffn = None
    if ff is None:
      unused.append(f"{p}.norm2")
    else:
      ffn = make(FEED_FORWARDS, "swiglu", f"{p}.mlp", W, ff, tensors=("gate", "up", "down"), activation="gelu_tanh")
    blocks.append(make(BLOCKS, "pre_norm", p, norm(f"{p}.norm1"), mixer, norm(f"{p}.norm2") if ffn is not None else None, ffn))
    run_list.append(LayerRun(i, cache_of))
  lm_head = LMHead("head", cfg.vocab, W, tensor="head")
  return ModelSpec(config=cfg, embedding=embedding, blocks=blocks, final_norm=norm("final.norm"), lm_head=lm_head,
                   position_encodings=list(encodings.values()), run_list=run_list, aliases={}, unused=unused,
                   init_std=cfg.initializer_range)
