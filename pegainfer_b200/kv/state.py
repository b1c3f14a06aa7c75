"""Per-request recurrent state in slots (slot 0 is the padding slot of CUDA-graph buckets).

``StateSlots`` is the slot bookkeeping: a request takes a slot at its first step and gives it back when it ends; a slot is
cleared when it is taken.  ``RecurrentState`` holds the state of models whose linear layers are all alike (one convolution
tensor and one state tensor over the layers), ``LayerStates`` that of models whose layers differ (a state tensor per layer,
and a convolution tensor where the layer has short convolutions).  A layer's state is f32 ``[slots, heads, dk, dv]``, its
carried convolution inputs ``[slots, channels, taps - 1]`` in the activation dtype.  The previous row that a token-shift mix
reads is kept as the carried input of a two-tap convolution; ``LayerStates.token`` (where the model's embedding looks at the
previous token) is int32 ``[slots]``, 1 + that token, 0 before the first.

Reference parity: pegainfer-qwen35/src/recurrent_state.rs:16-170.
"""
from __future__ import annotations

import torch


class StateSlots:
    def __init__(self, num_slots: int):
        self.num_slots = num_slots
        self._free = list(range(num_slots - 1, 0, -1))
        self.by_rid: dict = {}

    def clear(self, slot: int) -> None:
        raise NotImplementedError

    def slot_for(self, rid: int, fresh: bool) -> int:
        s = self.by_rid.get(rid)
        if s is None:
            if not self._free:
                raise RuntimeError("recurrent-state slot pool exhausted")
            s = self._free.pop()
            self.by_rid[rid] = s
            fresh = True
        if fresh:
            self.clear(s)
        return s

    def release(self, rid: int) -> None:
        s = self.by_rid.pop(rid, None)
        if s is not None:
            self._free.append(s)


class RecurrentState(StateSlots):
    def __init__(self, num_slots: int, n_linear: int, channels: int, conv_k: int, hv: int, dk: int, dv: int, dtype, device):
        super().__init__(num_slots)
        self.conv = torch.zeros((n_linear, num_slots, channels, conv_k - 1), dtype=dtype, device=device)
        self.ssm = torch.zeros((n_linear, num_slots, hv, dk, dv), dtype=torch.float32, device=device)

    def clear(self, slot: int) -> None:
        self.conv[:, slot].zero_()
        self.ssm[:, slot].zero_()


class LayerStates(StateSlots):
    def __init__(self, num_slots: int, geometries, dtype, device, token: bool = False):
        """``geometries``: ``(heads, dk, dv, conv_channels, taps)`` of every recurrent layer, ``taps == 0`` without
        short convolutions.  What a layer carries per channel in 32 bits is a state of ``dk == 1``; a layer may have several."""
        super().__init__(num_slots)
        self.token = torch.zeros(num_slots, dtype=torch.int32, device=device) if token else None
        self.ssm = [torch.zeros((num_slots, h, dk, dv), dtype=torch.float32, device=device) for h, dk, dv, _, _ in geometries]
        self.conv = [torch.zeros((num_slots, c, max(taps - 1, 0)), dtype=dtype, device=device) if taps else None for _, _, _, c, taps in geometries]

    def clear(self, slot: int) -> None:
        live = [t[slot] for t in (*self.ssm, *self.conv) if t is not None and t.numel()]
        if live:
            torch._foreach_zero_(live)
        if self.token is not None:
            self.token[slot].zero_()
