"""Korurax, put together from parts.

Per layer a pre-norm layer (layer norms with a weight and no bias) whose sublayers' outputs enter the residual stream times
``residual_mult``; what a layer hands on is a weighted sum of the embedding's rows and of every layer's result so far
(``DepthAverageBlock``).  The mixer is one of

  * ``latent_attention`` - attention through a latent with a rotated key part shared by all heads, without sink or gate
    (``LatentAttentionMixer`` with those options);
  * ``attention`` - grouped-query attention inside chunks of ``mask.size`` positions, without rotation: a distance bias
    ``r1 ln(1 + r2 d)`` per head is taken off the scores, a sink per head joins the softmax, and a gate per head multiplies
    its output (``GatedAttentionMixer`` with those options).

The feed-forward is a dense clamped gated one (``SwiGLUFeedForward`` with that activation), a mixture of squared-ReLU experts
chosen by their sigmoid scores, whose shares are multiplied with a constant (``RoutedExpertsFeedForward`` with those options), or
absent.  Around the layers: an embedding, a final layer norm, and the embedding table as the head, its logits capped by a tanh.
Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.dwa``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``.
"""

from __future__ import annotations

from ..config.model_config import KoruraxConfig
from ..config.registry import register_model
from ..parts import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, LMHead, TokenEmbedding, make
from .spec import ModelSpec


@register_model("Korurax", KoruraxConfig)
def build_korurax(cfg: KoruraxConfig) -> ModelSpec:
  W, eps, mult, n = cfg.width, cfg.norm_eps, float(cfg.residual_mult), len(cfg.layers)
  embedding = TokenEmbedding("embed", cfg.vocab, W, tensor="embed")
  blocks, encodings, unused = [], {}, []

  def rotary(rot):
    key = (rot.dims, rot.base)
    if key not in encodings:      # layers that rotate alike share a table
      encodings[key] = make(POSITION_ENCODINGS, "scaled_rotary", f"rot{len(encodings)}", rot.dims, rot.base, cfg.max_position_embeddings)
    return encodings[key]

  def norm(name):
    return make(NORMS, "layernorm", name, W, eps, weight_name=name, biased=False)

  for i in range(n):
    p = f"l{i}"
    m, mlp = cfg.mixer_of(i), cfg.mlp_of(i)
    if cfg.type_of(i) == "latent_attention":
      mixer = make(MIXERS, "latent_attention", f"{p}.mix", W, m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, eps,
                   rotary(m.rot), rotary_interleaved=False, sinks=False, gated=False)
    else:
      mixer = make(MIXERS, "gated_attention", f"{p}.mix", W, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, None, None, sinks=True,
                   gated=True, gate_per_head=True, chunk=m.chunk, distance_bias=True)
    if mlp is None:
      ffn = None
      unused.append(f"{p}.norm2")
    elif mlp.kind == "dense":
      ffn = make(FEED_FORWARDS, "swiglu", f"{p}.mlp", W, mlp.ff, tensors=("gate", "up", "down"), activation="clamped", limit=mlp.limit)
    else:
      ffn = make(FEED_FORWARDS, "routed_experts", f"{p}.mlp", W, mlp.ff, mlp.experts, mlp.top, router_weights="sigmoid_share",
                 activation="relu_squared", correction=False, weight_scale=mlp.scale)
    blocks.append(make(BLOCKS, "depth_average", p, i, n, W, norm(f"{p}.norm1"), mixer, norm(f"{p}.norm2") if ffn is not None else None, ffn,
                       mult=mult))
  final_norm = make(NORMS, "depth_average", "final", norm("final.norm"))
  lm_head = LMHead("head", cfg.vocab, W, tied_to=embedding, softcap=float(cfg.logit_softcap))
  return ModelSpec(config=cfg, embedding=embedding, blocks=blocks, final_norm=final_norm, lm_head=lm_head,
                   position_encodings=list(encodings.values()), aliases={}, unused=unused, init_std=cfg.initializer_range)
