"""Sapanex decoder: from its typed config to a :class:`ModelSpec`.

A layer norms the sum: x <- norm(alpha x + sublayer(x)), with the stream's own multiplier alpha (block kind
`sum_norm`).  A mixer is either grouped-query attention (`gqa_attention`: queries and keys normed over all heads'
rows at once, a partial half-split rotation whose frequencies are blended along a ramp, values turned by their own
position and the head's output turned back, a window of tokens beside the means of the blocks before it), or a
generalized delta rule (`general_delta`: a matrix state per head with a decay and a removal rate per key channel).
The feed-forward is relu squared between two matrices, or absent.  The output matrix is the token table, without the
embedding's multiplier.

Tensor names: `embed`, `final.norm`, and under `l<i>.`: `norm1`, `norm2`, `mix.{q,k,v,o,q.norm,k.norm}` or
`mix.{r,k,v,g,a,a.b,w0,w1,w2,norm,o}`, `mlp.{up,down}`.
"""
from __future__ import annotations

import math

from ..config.registry import Architecture
from ..config.sapanex import AttentionMixer, SapanexConfig
from ..config.spec import LayerSpec, ModelSpec, PartSpec

# The design fixes these: the recurrence's decay exp(-LOG_DECAY * sigmoid(..)) and what joins the sum of squares
# under a unit key's root.
LOG_DECAY = math.exp(-0.5)
UNIT_EPS = 1e-6


def build_spec(cfg: SapanexConfig) -> ModelSpec:
    norm = PartSpec.make("rms", eps=cfg.eps, weight_suffix="")
    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        if isinstance(m, AttentionMixer):
            position = values = PartSpec.make("none")
            if m.rot is not None:
                s = m.rot.scaling
                position = PartSpec.make("rope_neox", theta=m.rot.base, rotary_dim=m.rot.dims,
                                         ramp=None if s is None else (s.factor, s.original, s.fast, s.slow))
                values = PartSpec.make("rope_neox", theta=m.rot.base, rotary_dim=m.vdim)
            mixer = PartSpec.make(
                "gqa_attention", hidden_size=cfg.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim,
                v_head_dim=m.vdim, qk_norm="rows", qk_norm_eps=cfg.eps, scale=m.scale, max_positions=cfg.max_positions,
                position=position, value_position=values,
                window=None if m.mask is None else m.mask.size, pool=None if m.mask is None else m.mask.pool,
                names=(("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("qn", "q.norm"), ("kn", "k.norm")))
        else:
            mixer = PartSpec.make("general_delta", hidden_size=cfg.width, heads=m.heads, head_dim=m.dim, eps=cfg.eps,
                                  log_decay=LOG_DECAY, unit_eps=UNIT_EPS)
        ffn = PartSpec.make("none")
        if layer.ff:
            ffn = PartSpec.make("two_matrix", hidden_size=cfg.width, intermediate_size=layer.ff, activation="relu2",
                                names=(("up", "up"), ("down", "down")))
        block = PartSpec.make("sum_norm", hidden_size=cfg.width, alpha=cfg.alpha, mixer_prefix="mix.", ffn_prefix="mlp.",
                              mixer_norm="norm1", ffn_norm="norm2")
        layers.append(LayerSpec(prefix=f"l{i}.", block=block, mixer=mixer, feed_forward=ffn, norm=norm))
    return ModelSpec(
        architecture="Sapanex",
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        max_positions=cfg.max_positions,
        embedding_name="embed",
        head_name=None,
        final_norm_name="final.norm",
        final_norm=norm,
        layers=tuple(layers),
        weight_prefixes=("",),
        embedding_scale=cfg.embedding_scale,
    )


ARCHITECTURE = Architecture(
    name="sapanex",
    claims=("Sapanex", "sapanex"),
    read_config=SapanexConfig.from_dict,
    build_spec=build_spec,
)
