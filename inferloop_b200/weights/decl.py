"""What a part says about each tensor it needs."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Tuple


class FreeDim(int):
    """A dimension that the configuration does not give: the stored tensor decides it.  All dimensions of one
    `name` must agree within a model; the number itself is what random weights are made with."""

    name: str

    def __new__(cls, size: int, name: str) -> "FreeDim":
        self = super().__new__(cls, size)
        self.name = name
        return self


def shapes_agree(declared, stored, found) -> bool:
    """Whether a stored shape is the declared one.  `found` remembers what each free dimension turned out to be."""
    if len(declared) != len(stored):
        return False
    for d, s in zip(declared, stored):
        if isinstance(d, FreeDim):
            if s <= 0 or found.setdefault(d.name, int(s)) != s:
                return False
        elif d != s:
            return False
    return True


@dataclass(frozen=True)
class WeightDecl:
    """One tensor a part needs, by name.  A dimension of `shape` may be a :class:`FreeDim`.

    role:  "matrix" and "table" follow the engine's compute dtype (bfloat16, or float32
           on the 32-bit path); "vector" (norm weights, biases) is held in float32, which
           keeps a 32-bit tensor as stored and widens a 16-bit one without loss;
           "int" is an integer table held as int32.
    init:  distribution used by the random-weights mode: "normal" N(0, 0.02),
           "norm" 1 + N(0, 0.1), "bias" N(0, 0.02), "mix" 0.5 + N(0, 0.1), "eye" identity + N(0, 0.1), "around_zero" N(0, 0.1), "decay" N(0, 0.7), "positive" 0.02 + |N(0, 0.1)|, "zeros".
    root:  True when the name is not under the model's weight prefix
           (`lm_head.weight`, crates/foundation/spi/src/model.rs:220-226).
    optional: a tensor that a file may hold although the model does not read it (or may leave
           out): it is neither missing nor unexpected, and is not bound when absent.
    """

    name: str
    shape: Tuple[int, ...]
    role: str = "matrix"
    init: str = "normal"
    root: bool = False
    optional: bool = False

    def under(self, prefix: str) -> "WeightDecl":
        if self.root:
            return self
        return WeightDecl(prefix + self.name, self.shape, self.role, self.init, self.root, self.optional)
