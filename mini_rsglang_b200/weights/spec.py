"""What a part asks of a checkpoint: one `WeightSpec` per tensor."""
from __future__ import annotations

from dataclasses import dataclass


@dataclass(frozen=True)
class WeightSpec:
    """`role` decides the dtype the tensor is held in and how random weights draw it:
    - "matrix": a projection or table of activations' kind; held in the engine's dtype
      (bfloat16 when serving, float32 on the 32-bit path); drawn N(0, 0.02);
    - "vector": a norm's scale; always held in float32 (widening bfloat16 is exact, a tensor
      stored in 32-bit stays so); drawn 1 + N(0, 0.05);
    - "offset_vector": a norm's scale stored as its distance from one; held in float32; drawn N(0, 0.05);
    - "bias": a bias, a small table or a constant of a recurrence, wanted in full precision; always held in
      float32; drawn N(0, 0.5);
    - "int_table": integers; held as int32.
    A size of -1 in `shape` stands for "whatever the checkpoint has" (a table whose length only the file states);
    seeded random weights cannot be drawn for such a spec.
    `optional_skip` names a tensor that may be present but is not used (a tied head)."""

    name: str
    shape: tuple[int, ...]
    role: str = "matrix"
