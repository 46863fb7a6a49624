"""Small Tamovik configurations for the tests, their model folders and plain logits."""
from __future__ import annotations

import os
import random
from typing import Dict, List

import torch

import plain_tamovik as plain


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, scaling=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": m}


def parallel(left, right):
    """left = (heads, kv_heads, dim, conv, scale, chunk or None), right = (heads, dim, vdim, gate_cap)."""
    a = dict(zip(("heads", "kv_heads", "dim", "conv", "scale"), left))
    a["vdim"] = a["dim"]
    if left[5] is not None:
        a["mask"] = {"size": left[5]}
    return {"type": "parallel", "mixer": {"left": a, "right": dict(zip(("heads", "dim", "vdim", "gate_cap"), right))}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, groups=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": router, "expert": {"ff": ff, "limit": limit}}


def model(vocab, width, eps, layers, bigram=None):
    c = {"architecture": "Tamovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": [dict(l, mlp=f) for l, f in layers]}
    if bigram is not None:
        c["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    return c


# K: odd sizes, exact kernels only: groups of three heads, five taps, chunks of 13 positions over pages of 4, a state of 10 x 7,
# blended frequencies and plain ones, experts in three groups of which two stay, experts without groups, a layer without
# feed-forward.
CONFIG_K = model(203, 72, 1e-5, [
    (latent(3, 10, 6, 7, 20, 0.3, 40.0, (4.0, 60.0, 8.0, 1.0)), dense(52)),
    (parallel((6, 2, 12, 5, 0.4, 13), (3, 10, 7, 4.0)), moe(6, 2, 20, 0.8, groups=(3, 2))),
    (parallel((3, 3, 6, 2, 0.6, 30), (1, 5, 20, 9.0)), None),
    (latent(5, 6, 4, 12, 9, 0.5, 3000.0), moe(3, 3, 16, 2.5)),
], bigram=(101, 13, 5))
# L: the sizes the tensor-core kernels take: latent rows of 128 and of 64, heads of 64 and of 128 in chunks of 40 and 64 over pages
# of 16, states of 64 x 64 and 128 x 96; experts of 64 and 128 (the grouped tcgen05 product), four groups of which one stays.
CONFIG_L = model(1000, 256, 1e-6, [
    (latent(4, 64, 32, 64, 96, 0.1, 500000.0, (8.0, 256.0, 16.0, 1.0)), dense(512)),
    (parallel((8, 2, 64, 4, 0.125, 40), (4, 64, 64, 12.0)), moe(8, 2, 64, 1.0, groups=(4, 1))),
    (latent(8, 32, 16, 48, 48, 0.15, 10000.0), moe(4, 1, 128, 7.0)),
    (parallel((2, 1, 128, 3, 0.09, 64), (2, 128, 96, 15.0)), moe(12, 3, 64, 2.0, groups=(3, 2))),
], bigram=(509, 31, 3))
# M: everything another model makes plural is one: one head, one kv head, one tap, chunks of the token itself, a state of 1 x 1,
# one expert in one group, one bucket; a part of a single pair; sizes that are multiples of nothing.
CONFIG_M = model(101, 50, 3e-6, [
    (latent(1, 1, 2, 3, 5, 1.0, 7.0), moe(1, 1, 11, 1.0, groups=(1, 1))),
    (parallel((1, 1, 7, 1, 1.0, 1), (1, 1, 1, 1.0)), dense(13)),
    (parallel((1, 1, 9, 3, 0.7, 2), (1, 3, 5, 2.0)), dense(17)),
], bigram=(1, 1, 0))
# N: no latent layer, no second table, no chunks (every earlier key is seen): long-reaching left sides beside the memory.
CONFIG_N = model(150, 64, 1e-5, [
    (parallel((4, 1, 16, 2, 0.5, None), (2, 16, 33, 6.0)), moe(4, 2, 32, 1.5, groups=(2, 1))),
    (parallel((2, 2, 64, 4, 0.125, None), (3, 24, 8, 20.0)), dense(64)),
])
# P: cached rows of more than 512 elements, a state of 256 rows, one group of 20 heads in chunks longer than a page of 32.
CONFIG_P = model(500, 128, 2e-6, [
    (latent(3, 40, 64, 24, 520, 0.1, 30000.0, (40.0, 4096.0, 32.0, 1.0)), dense(192)),
    (parallel((20, 1, 32, 4, 0.2, 50), (1, 256, 80, 10.0)), moe(20, 4, 64, 3.0, groups=(5, 2))),
], bigram=(97, 7, 11))
CASES = {"K": (CONFIG_K, 51, 4), "L": (CONFIG_L, 52, 16), "M": (CONFIG_M, 53, 8), "N": (CONFIG_N, 54, 16), "P": (CONFIG_P, 55, 32)}   # config, seed, page size

_FOLDERS: Dict[tuple, str] = {}
_PLAIN: Dict[tuple, "Plain"] = {}


def _sharpen(name: str, t: torch.Tensor) -> torch.Tensor:
    """Random weights as the initialisers give them hide some faults: softmaxes that are flat, gates that hardly move, states that
    forget within a few tokens, routers that barely prefer an expert, corrections that never change the order.  Spread them."""
    n = t.numel()
    x = t.float()
    if name.endswith(".router"):
        return x * 8.0
    if name.endswith(".correction"):                # some scores far below zero: a choice score can be negative
        return (torch.linspace(-0.15, 0.15, n) - (0.8 if n > 1 else 0.0)).flip(0).view(t.shape)
    if name.endswith((".q.conv", ".k.conv")):       # taps of both signs, none of them alike
        return x + torch.linspace(-0.8, 0.6, t.shape[1])[None, :]
    if name.endswith((".left.q.norm", ".left.k.norm")):
        return x * 2.0
    if name.endswith(".left.g"):
        return x * 6.0
    if name.endswith((".right.i", ".right.f")):     # gates that depend on the input
        return x * 6.0
    if name.endswith(".right.f.b"):                 # from a few tokens to hundreds
        return torch.linspace(1.0, 5.0, n).view(t.shape)
    if name.endswith(".right.i.b"):
        return torch.linspace(-2.0, 2.0, n).view(t.shape) if n > 1 else x
    if name.endswith((".mix.q", ".mix.dkv", ".mix.uk", ".right.q", ".right.k", ".right.v")):
        return x * 3.0
    if name in ("embed", "bigram"):
        return x * 20.0
    if name == "head":
        return x * 6.0
    return t


def folder(tmp_root: str, name: str, dtype: torch.dtype) -> str:
    """The model folder of a case (weights stored in `dtype`), written once per test session."""
    from inferloop_b200.weights import write_random_model, write_safetensors
    from inferloop_b200.weights.safetensors_io import SafetensorsFile
    key = (name, dtype)
    if key not in _FOLDERS:
        config, seed, _ = CASES[name]
        path = os.path.join(tmp_root, f"tamovik-{name}-{str(dtype).split('.')[-1]}")
        write_random_model(path, config, seed, dtype, prefix="")
        f = SafetensorsFile(os.path.join(path, "model.safetensors"))
        tensors = [(n, f.tensor(n).clone()) for n in f.names()]
        f.close()
        made = {n: _sharpen(n, t) for n, t in tensors}
        for n in made:
            # A memory that holds one token gives v (k . q), normed: where k . q happens to cancel, its sign is decided by
            # rounding.  Queries near the keys keep every read-out away from that.
            if n.endswith(".right.q"):
                made[n] = 0.8 * made[n[:-1] + "k"] + 0.3 * made[n]
        tensors = [(n, made[n].to(t.dtype)) for n, t in tensors]
        write_safetensors(os.path.join(path, "model.safetensors"), tensors, metadata={"format": "pt"})
        _FOLDERS[key] = path
    return _FOLDERS[key]


class Plain:
    def __init__(self, config: dict, weights: Dict[str, torch.Tensor]) -> None:
        self.config = config
        self.w = {k: v.double() for k, v in weights.items()}

    def forward(self, tokens, trace=None) -> torch.Tensor:
        return plain.forward(self.w, self.config, list(tokens), trace)

    def least_margin(self, tokens, first: int = 0) -> float:
        """The smallest routing margin over the positions from `first` on, in every routed layer."""
        margins: List[torch.Tensor] = []
        plain.forward(self.w, self.config, list(tokens), margins=margins)
        return min([1.0] + [float(m[first:].min()) for m in margins])


def plain_model(tmp_root: str, name: str, dtype: torch.dtype) -> Plain:
    from inferloop_b200.weights.safetensors_io import SafetensorsFile
    key = (name, dtype)
    if key not in _PLAIN:
        path = folder(tmp_root, name, dtype)
        f = SafetensorsFile(os.path.join(path, "model.safetensors"))
        weights = {n: f.tensor(n).clone() for n in f.names()}
        f.close()
        _PLAIN[key] = Plain(CASES[name][0], weights)
    return _PLAIN[key]


def decided_tokens(model: Plain, n: int, vocab: int, seed: int, margin: float, chunk: int = 12) -> List[int]:
    """`n` random tokens whose routing decisions, in the plain model, all have at least this margin, so that no comparison
    rests on a close call.  The sequence grows by chunks; a chunk whose positions are not all decided is drawn again."""
    rng = random.Random(seed)
    tokens: List[int] = []
    failed = 0
    while len(tokens) < n:
        size = max(1, chunk >> (failed // 3))
        more = [rng.randrange(vocab) for _ in range(min(size, n - len(tokens)))]
        if model.least_margin(tokens + more, len(tokens)) >= margin:
            tokens += more
            failed = 0
        else:
            failed += 1
            if failed > 400:
                raise AssertionError("no token sequence with decided routing found")
    return tokens
