"""Maps between a sublayer's norm and the sublayer.

``residual_conv``: a short causal convolution per channel over time, added to its input,

    y_t = x_t + sum_j w[:, j] x_(t - taps + 1 + j),   zeros before the sequence's start

with w [D, taps] and no bias.  State per request: the last taps - 1 inputs x (float32, in a slot).  Behind a
norm that offers `Norm.group_prologue` it runs inside the launch that folds the stream and norms it
(csrc/fold_norm.cu), on the float normed rows; behind any other norm as a launch of its own over the stored rows.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..kernels import ops as K
from .base import InputMap, ParamSpec, StateSpec, register_input_map

Tensor = torch.Tensor


class ResidualConv(InputMap):
    def __init__(self, hidden_size: int, taps: int, tensor: str = ""):
        if taps < 1:
            raise ValueError("the convolution needs at least one tap")
        self.hidden_size, self.taps, self.tensor = int(hidden_size), int(taps), str(tensor)

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec(self.tensor, (self.hidden_size, self.taps), kind="vector", init=("normal", 0.3))]

    def state_specs(self) -> List[StateSpec]:
        return [StateSpec.fixed("inputs", (self.taps - 1, self.hidden_size), "float32")] if self.taps > 1 else []

    def bind(self, params: Dict[str, Tensor]) -> None:
        w = params[self.tensor]
        self.taps_t = w.t().contiguous()
        # as a launch of its own: the input itself is one more on the current token's tap
        self.w_own = w.clone()
        self.w_own[:, -1] += 1.0
        self.w_own_t = self.w_own.t().contiguous()
        self.ones = torch.ones(self.hidden_size, dtype=torch.float32, device=w.device)

    def _window(self, cache):
        return cache.fixed(f"{self.name}.inputs") if self.taps > 1 else None

    def fused_conv(self, cache):
        return self.taps_t, self._window(cache)

    def forward(self, x: Tensor, ctx, cache, out: Tensor) -> None:
        window = self._window(cache)
        if window is None:
            window = torch.empty((0, 0, self.hidden_size), dtype=torch.float32, device=x.device)
        if ctx.decode_only:
            K.conv1d_decode(x, self.ones, None, self.w_own, None, window, ctx.slots, out, activation=False)
            return
        K.conv1d_fwd(x, self.ones, None, self.w_own, None, window, ctx.seq_of, ctx.cu_seqlens, ctx.slots, out,
                     weight_t=self.w_own_t, activation=False)
        K.conv1d_window_update(x, self.ones, None, window, ctx.cu_seqlens, ctx.slots, ctx.n_seq, self.taps)


register_input_map("residual_conv", ResidualConv)
