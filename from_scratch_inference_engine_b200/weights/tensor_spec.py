"""What a part says about each tensor it needs."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Sequence, Tuple


@dataclass(frozen=True)
class TensorSpec:
    """One named tensor of a checkpoint.

    role      "matrix": operand of a matrix product, held in the compute dtype;
              "vector": gain or bias, a tensor stored in 32-bit stays in 32-bit;
              "table":  integer table, held as int32.
    init      how the random-weights mode draws it: "normal" (N(0, std)),
              "gain" (1 + N(0, std)), "zeros", "ones", "taps" (N(0, 0.5): the taps of a short
              convolution, whose scale a norm behind it removes), "half" (1/2 + N(0, std): a blending
              weight) or "eye" (identity + N(0, std):
              a matrix that mixes heads).
    optional  may be absent from the checkpoint (the part says what it does then).
    free      dimensions whose size the checkpoint decides (a size that no configuration key gives);
              `shape` then holds what the random-weights mode draws.
    same_as   when present in the checkpoint it must equal this other tensor
              (a head tied to the embedding that is stored a second time).
    """

    name: str
    shape: Tuple[int, ...]
    role: str = "matrix"
    init: str = "normal"
    optional: bool = False
    same_as: str = ""
    free: Tuple[int, ...] = ()

    def fits(self, shape: Sequence[int]) -> bool:
        """Whether a stored tensor of `shape` is one of this kind."""
        return len(shape) == len(self.shape) and all(
            have == want or (axis in self.free and have > 0)
            for axis, (have, want) in enumerate(zip(shape, self.shape)))
