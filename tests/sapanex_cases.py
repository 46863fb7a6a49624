"""Small Sapanex configurations for the tests, their model folders and plain logits."""
from __future__ import annotations

import math
import os
from typing import Dict

import torch

import plain_sapanex as plain


def attention(heads, kv_heads, dim, vdim, scale, rot=None, mask=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        base, dims, scaling = rot
        m["rot"] = {"base": base, "dims": dims}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if mask is not None:
        m["mask"] = {"size": mask[0], "pool": mask[1]}
    return m


def layer(mixer, ff):
    return {"type": "attention" if "kv_heads" in mixer else "general_delta", "mixer": mixer,
            "mlp": None if not ff else {"kind": "dense", "ff": ff}}


def delta(heads, dim):
    return {"heads": heads, "dim": dim}


def model(vocab, width, eps, scale, alpha, layers):
    return {"architecture": "Sapanex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "postln_alpha": alpha, "layers": layers}


# K: odd sizes, exact kernels only.  Groups of five heads, values narrower and wider than keys, a rotation of part of a head
# whose ramp meets kept, blended and divided pairs, blocks shorter and longer than the window, layers with and without
# feed-forward, heads of the recurrence that fill no multiple of anything.
CONFIG_K = model(203, 72, 1e-5, 2.5, 1.7, [
    layer(delta(3, 10), 40),
    layer(attention(5, 1, 12, 10, 0.5, rot=(30.0, 8, (4.0, 60, 8.0, 1.0)), mask=(7, 3)), 36),
    layer(delta(1, 20), 0),
    layer(attention(4, 4, 6, 14, 0.9, rot=(100.0, 4, None), mask=(5, 9)), 0),
])
# L: the sizes the tensor-core kernels take: heads of 64 / 64, 128 / 64 and 128 / 128; states of 64 x 64 and 128 x 128.
CONFIG_L = model(1000, 256, 1e-6, 0.75, 2.2, [
    layer(attention(8, 2, 64, 64, 0.2, rot=(10000.0, 64, (8.0, 256, 16.0, 1.0)), mask=(50, 8)), 512),
    layer(delta(2, 64), 0),
    layer(attention(4, 1, 128, 64, 0.15, rot=(500000.0, 32, None), mask=(20, 4)), 256),
    layer(delta(2, 128), 384),
    layer(attention(2, 2, 128, 128, 0.15, rot=(3000.0, 128, (2.0, 64, 4.0, 0.5)), mask=(33, 1)), 0),
])
# M: sizes that are multiples of nothing, and everything another model makes plural is one: one head, one kv head, a window of the token itself, a rotation of a single pair.
CONFIG_M = model(101, 50, 3e-6, 1.0, 3.0, [
    layer(attention(1, 1, 7, 6, 0.8, rot=(3.0, 2, None), mask=(1, 2)), 13),
    layer(delta(1, 9), 11),
    layer(delta(2, 7), 0),
])
# N: recurrences only: no pages, only state slots.
CONFIG_N = model(150, 64, 1e-5, 1.5, 3.5, [layer(delta(2, 32), 96), layer(delta(4, 16), 0), layer(delta(1, 160), 64)])
# O: attention only, a layer without a window (every earlier token, values turned all the same) and one without any rotation.
CONFIG_O = model(170, 96, 2e-5, 1.25, 1.4, [
    layer(attention(6, 3, 32, 16, 0.3, rot=(500.0, 16, (16.0, 32, 32.0, 2.0))), 80),
    layer(attention(3, 3, 64, 64, 0.15, rot=(900.0, 24, None)), 0),
    layer(attention(2, 1, 24, 20, 0.4, mask=(11, 4)), 48),
])
# P: groups of 32 and 20 query heads on one key head (more than the decode kernel merges in one pass), pages of 32 and blocks that do not
# divide a page.
CONFIG_P = model(300, 128, 1e-6, 0.9, 2.0, [
    layer(attention(32, 1, 64, 64, 0.2, rot=(20000.0, 32, (4.0, 128, 8.0, 1.0)), mask=(70, 5)), 0),
    layer(delta(3, 48), 192),
    layer(attention(20, 1, 128, 64, 0.12, rot=(700.0, 64, None), mask=(40, 24)), 128),
])
CASES = {"K": (CONFIG_K, 61, 4, 5), "L": (CONFIG_L, 62, 16, 24), "M": (CONFIG_M, 63, 8, 1), "N": (CONFIG_N, 64, 16, 13), "O": (CONFIG_O, 65, 8, 1),
         "P": (CONFIG_P, 66, 32, 40)}     # config, seed, page size, inner size of the decays' map

_FOLDERS: Dict[tuple, str] = {}
_PLAIN: Dict[tuple, "Plain"] = {}


def _sharpen(name: str, t: torch.Tensor) -> torch.Tensor:
    """Random weights as the initialisers give them hide some faults: products close to zero, decays all alike, a softmax that
    averages.  Spread them: products of unit gain, decays from a token to thousands, removal rates from none to all."""
    n = t.numel()
    if name == "embed":
        return t.float() * 40.0
    if name.endswith(".w0"):
        return torch.linspace(-9.0, 2.0, n).view(t.shape)
    if name.endswith(".a.b"):
        return torch.linspace(-4.0, 3.0, n).flip(0).view(t.shape)
    if t.dim() == 2:
        return t.float() / (0.02 * math.sqrt(t.shape[1]))
    return t


def folder(tmp_root: str, name: str, dtype: torch.dtype) -> str:
    """The model folder of a case (weights stored in `dtype`), written once per test session.  The inner size of the decays'
    map, which the configuration does not give, is the case's own."""
    from inferloop_b200.weights import write_random_model, write_safetensors
    from inferloop_b200.weights.decl import WeightDecl
    from inferloop_b200.weights.random_init import random_tensor
    from inferloop_b200.weights.safetensors_io import SafetensorsFile
    key = (name, dtype)
    if key not in _FOLDERS:
        config, seed, _, rank = CASES[name]
        path = os.path.join(tmp_root, f"sapanex-{name}-{str(dtype).split('.')[-1]}")
        write_random_model(path, config, seed, dtype, prefix="")
        f = SafetensorsFile(os.path.join(path, "model.safetensors"))
        tensors = [(n, f.tensor(n).clone()) for n in f.names()]
        f.close()
        out = []
        for n, t in tensors:
            if n.endswith(".w1"):
                t = random_tensor(WeightDecl(n, (rank, t.shape[1])), seed, dtype)
            if n.endswith(".w2"):
                t = random_tensor(WeightDecl(n, (t.shape[0], rank)), seed, dtype)
            out.append((n, _sharpen(n, t).to(t.dtype)))
        write_safetensors(os.path.join(path, "model.safetensors"), out, metadata={"format": "pt"})
        _FOLDERS[key] = path
    return _FOLDERS[key]


class Plain:
    def __init__(self, config: dict, weights: Dict[str, torch.Tensor]) -> None:
        self.config = config
        self.w = {k: v.double() for k, v in weights.items()}
        self._kept: Dict[tuple, torch.Tensor] = {}

    def forward(self, tokens, trace=None) -> torch.Tensor:
        key = tuple(tokens)
        if trace is not None or key not in self._kept:
            out = plain.forward(self.w, self.config, list(tokens), trace)
            if trace is not None:
                return out
            self._kept[key] = out
        return self._kept[key]


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
