"""Tamovik decoder: from its typed config to a :class:`ModelSpec`.

The embedding is the token's row plus a row of a second table chosen by the pair of the previous token and the token.  A
layer norms what its sublayers give (block kind `output_norm`).  A mixer is either attention over a cached latent with a
rotated key part shared by all heads (`latent_attention` with `rot_dim`; pairs half of the part apart, frequencies blended
along a ramp), or two mixers side by side whose outputs are each normed over the width and averaged (`parallel` with
`out_norms`): grouped-query attention inside aligned chunks, without positions, whose queries and keys pass a short
convolution and a norm over whole rows, whose values are the convolved keys and whose output is gated element by element
(`gqa_attention` with `chunk`, `conv`, `values`, `output_gate`), beside a matrix memory (`mlstm`).  The feed-forward is a
gated unit with gelu, or routed experts (sigmoid scores, a correction that only ranks, groups ranked by their two best
members, weights as they are) with the clamped gated unit, or absent.  The output matrix is a tensor of its own.

Tensor names: `embed`, `bigram`, `final.norm`, `head`, and under `l<i>.`: `norm1`, `norm2`,
`mix.{q,dkv,dkv.norm,uk,uv,o}`, or `mix.left.{q,k,q.conv,k.conv,q.norm,k.norm,g,o,out}` with
`mix.right.{q,k,v,g,i,i.b,f,f.b,norm,o,out}`; `mlp.{gate,up,down}` or `mlp.router`, `mlp.correction`,
`mlp.e<j>.{gate,up,down}`.
"""
from __future__ import annotations

from ..config.registry import Architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec
from ..config.tamovik import DenseFeedForward, LatentMixer, TamovikConfig

# The design fixes these: the experts' gate a(g) = g * sigmoid(1.702 g) and the one added to its clamped linear half; what
# joins the matrix memory's denominator; the mean of the two branches.
GATE_SHARPNESS = 1.702
UP_OFFSET = 1.0
DENOMINATOR_EPS = 1e-6
BRANCH_MULT = 0.5

GLU_NAMES = (("gate", "gate"), ("up", "up"), ("down", "down"))


def build_spec(cfg: TamovikConfig) -> ModelSpec:
    norm = PartSpec.make("rms", eps=cfg.eps, weight_suffix="")
    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        if isinstance(m, LatentMixer):
            position = None
            if m.rot is not None:
                s = m.rot.scaling
                position = PartSpec.make("rope_neox", theta=m.rot.base, rotary_dim=m.rot.dims,
                                         ramp=None if s is None else (s.factor, s.original, s.fast, s.slow))
            mixer = PartSpec.make(
                "latent_attention", hidden_size=cfg.width, heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim, latent=m.kv_rank,
                scale=m.scale, eps=cfg.eps, max_positions=cfg.max_positions, rot_dim=m.rot_dim, position=position)
        else:
            a, b = m.left, m.right
            left = PartSpec.make(
                "gqa_attention", hidden_size=cfg.width, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.dim,
                qk_norm="rows", qk_norm_eps=cfg.eps, scale=a.scale, max_positions=cfg.max_positions, position=PartSpec.make("none"),
                chunk=a.chunk, conv=a.conv, values="keys", output_gate="element",
                names=(("q", "q"), ("k", "k"), ("o", "o"), ("g", "g"), ("qc", "q.conv"), ("kc", "k.conv"), ("qn", "q.norm"), ("kn", "k.norm")))
            right = PartSpec.make("mlstm", hidden_size=cfg.width, heads=b.heads, head_dim=b.dim, v_head_dim=b.vdim, eps=cfg.eps,
                                  gate_cap=b.gate_cap, den_eps=DENOMINATOR_EPS)
            mixer = PartSpec.make("parallel", hidden_size=cfg.width, branches=(("left.", left), ("right.", right)),
                                  out_norms=("left.out", "right.out"), norm_eps=cfg.eps, out_mult=BRANCH_MULT)
        f = layer.mlp
        if f is None:
            ffn = PartSpec.make("none")
        elif isinstance(f, DenseFeedForward):
            ffn = PartSpec.make("swiglu", hidden_size=cfg.width, intermediate_size=f.ff, activation="gelu_tanh", names=GLU_NAMES)
        else:
            ffn = PartSpec.make(
                "routed_experts", hidden_size=cfg.width, experts=f.experts, top_k=f.top, expert_inter=f.ff, score="sigmoid",
                renormalize=False, weight_on="output", correction=True, groups=(f.groups, f.keep) if f.groups > 1 else None,
                group_rank="best_two",
                activation=PartSpec.make("clamped_glu", limit=f.limit, sharpness=GATE_SHARPNESS, up_offset=UP_OFFSET),
                names=(("router", "router"), ("correction", "correction"), ("gate", "e{e}.gate"), ("up", "e{e}.up"), ("down", "e{e}.down")))
        block = PartSpec.make("output_norm", hidden_size=cfg.width, mixer_prefix="mix.", ffn_prefix="mlp.", mixer_norm="norm1",
                              ffn_norm="norm2")
        layers.append(LayerSpec(prefix=f"l{i}.", block=block, mixer=mixer, feed_forward=ffn, norm=norm))
    embedding = None
    if cfg.pairs is not None:
        embedding = PartSpec.make("hashed_pairs", hidden_size=cfg.width, buckets=cfg.pairs.buckets, mul_prev=cfg.pairs.mul_prev,
                                  mul_cur=cfg.pairs.mul_cur, table="bigram")
    return ModelSpec(
        architecture="Tamovik",
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        max_positions=cfg.max_positions,
        embedding_name="embed",
        head_name="head",
        final_norm_name="final.norm",
        final_norm=norm,
        layers=tuple(layers),
        weight_prefixes=("",),
        embedding=embedding,
    )


ARCHITECTURE = Architecture(
    name="tamovik",
    claims=("Tamovik", "tamovik"),
    read_config=TamovikConfig.from_dict,
    build_spec=build_spec,
)
