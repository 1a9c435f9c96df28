"""Per-sequence recurrent state of the running sequences, one slot each.

KV pages grow with a sequence; state does not.  The scheduler hands every running sequence one slot
(csrc/runtime/core.h ``num_state_slots``) and the step plan carries it beside the page-table row.  A slot is never
cleared: kernels start from zero when a sequence's rows begin at position 0.
"""
from __future__ import annotations

import torch


class StateCache:
    def __init__(self, cfg, slots: int, device):
        self.slots = slots
        self.layers = [{name: torch.zeros(slots, *shape, dtype=torch.float32, device=device) for name, shape in cfg.state_shapes(li).items()}
                       for li in range(cfg.num_layers)]

    def nbytes(self) -> int:
        return sum(t.numel() * 4 for layer in self.layers for t in layer.values())
