"""Mamba-1: a selective scan whose decay is a table over channels and state entries.

    [x | z] = W_in u (inner each);  x <- silu(conv(x) + b), a causal convolution per channel;
    [t | B | C] = W_x x (dt_rank, state, state);  dt = softplus(W_dt t + b_dt), one per channel;
    A = -exp(A_log) [inner, state];
    S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c;
    out = W_o (y * silu(z)).

State per request (float32, in a slot, zero for a new request): S [inner, state] and the last taps - 1 inputs of
the convolution.  The step sizes, decays, the state and its read-out are float arithmetic in both storage
types; the projections, the convolution and the gate have the storage type.  W_x is stored with zero rows
behind the step sizes' rows and at its end, so that t, B and C start on 16-byte boundaries, and W_dt with zero
columns to match.  A decode step of few requests makes W_dt t inside the scan's launch.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..kernels import ops as K
from . import branches, streaming
from .base import ParamSpec, StateSpec, register_mixer
from .recurrent import _StackedInput

Tensor = torch.Tensor


# From this many (request, rank) products on, a decode step makes its step sizes by a product of their own: every
# request of the scan's launch would read W_dt again.  Measured (us, in the launch / product and launch): 16 requests of
# 6,144 channels and rank 192 9.9 / 8.0, 8 of them 6.4 / 6.0; 32 requests of 2,048 channels and rank 64 5.4 / 6.2, 64 of
# them 9.0 / 9.0.
_OWN_PRODUCT_FROM = 2560


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


class SelectiveScanMixer(_StackedInput):
    def __init__(self, hidden_size: int, inner: int, state: int, dt_rank: int, conv: int, out_multiplier: float = 1.0):
        if min(inner, state, dt_rank, conv) < 1:
            raise ValueError("inner, state, dt_rank and conv must be positive")
        if state > K.SELECTIVE_MAX_STATE:
            raise ValueError(f"the scan kernels take state sizes up to {K.SELECTIVE_MAX_STATE}, got {state}")
        self.hidden_size = int(hidden_size)
        self.inner, self.d_state, self.dt_rank, self.taps = int(inner), int(state), int(dt_rank), int(conv)
        self.out_scale = float(out_multiplier)
        self.rank_padded = _up8(self.dt_rank)
        self.off_b = self.rank_padded
        self.off_c = self.off_b + _up8(self.d_state)
        self.low_rows = self.off_c + _up8(self.d_state)

    def param_specs(self) -> List[ParamSpec]:
        D, I, N, R = self.hidden_size, self.inner, self.d_state, self.dt_rank
        return [ParamSpec("in", (2 * I, D)),
                ParamSpec("conv", (I, self.taps), kind="vector", init=("normal", 0.5)),
                ParamSpec("conv.b", (I,), kind="vector", init=("normal", 0.1)),
                ParamSpec("x", (R + 2 * N, I), init=("normal", 0.05)),
                ParamSpec("dt", (I, R), init=("normal", 0.2)),
                ParamSpec("dt.b", (I,), kind="vector", init=("inv_softplus_log_uniform", 1e-3, 0.1)),
                ParamSpec("A_log", (I, N), kind="vector", init=("log_uniform", 1.0, 16.0)),
                ParamSpec("D", (I,), kind="vector", init=("ones",)),
                ParamSpec("o", (D, I))]

    def state_specs(self) -> List[StateSpec]:
        return [StateSpec.fixed("conv", (self.taps - 1, self.inner), "float32"),
                StateSpec.fixed("S", (self.inner, self.d_state), "float32")]

    def bind(self, params: Dict[str, Tensor]) -> None:
        I, N, R = self.inner, self.d_state, self.dt_rank
        self.w_in = params["in"].contiguous()
        self.w_out = params["o"].contiguous()
        self.conv_w = params["conv"].contiguous()
        self.conv_w_t = self.conv_w.t().contiguous()
        self.conv_b = params["conv.b"].contiguous()
        self.conv_ones = torch.ones(I, dtype=torch.float32, device=self.conv_w.device)
        w_x = params["x"]
        self.w_x = torch.zeros((self.low_rows, I), dtype=w_x.dtype, device=w_x.device)
        self.w_x[:R] = w_x[:R]
        self.w_x[self.off_b:self.off_b + N] = w_x[R:R + N]
        self.w_x[self.off_c:self.off_c + N] = w_x[R + N:]
        self.w_dt = torch.zeros((I, self.rank_padded), dtype=w_x.dtype, device=w_x.device)
        self.w_dt[:, :R] = params["dt"]
        self.dt_bias, self.d_skip = params["dt.b"].contiguous(), params["D"].contiguous()
        self.a_log = params["A_log"].contiguous()

    def output_weight(self) -> Tensor:
        return self.w_out

    def forward_projected(self, proj: Tensor, ctx, cache, out: Tensor) -> None:
        streaming.linear(self.pre_output(proj, ctx, cache), self.w_out, out, ctx)

    def pre_output(self, proj: Tensor, ctx, cache) -> Tensor:
        T, I, ws = proj.shape[0], self.inner, ctx.workspace
        raw_x, z = proj[:, :I], proj[:, I:2 * I]
        window, state = cache.fixed(f"{self.name}.conv"), cache.fixed(f"{self.name}.S")
        x = ws.alloc((T, I), proj.dtype)
        low = ws.alloc((T, self.low_rows), proj.dtype)
        y = ws.alloc((T, I), proj.dtype)
        if ctx.decode_only:
            K.conv1d_decode(raw_x, self.conv_ones, None, self.conv_w, self.conv_b, window, ctx.slots, x)
            streaming.linear(x, self.w_x, low, ctx)
            raw_dt = None
            if T * self.dt_rank >= _OWN_PRODUCT_FROM:
                raw_dt = ws.alloc((T, I), proj.dtype)
                streaming.linear(low[:, :self.rank_padded], self.w_dt, raw_dt, ctx)
            K.selective_step(x, low, self.rank_padded, self.off_b, self.off_c, self.w_dt, z, self.dt_bias, self.a_log,
                             self.d_skip, state, ctx.slots, y, raw=raw_dt)
            return y
        K.conv1d_fwd(raw_x, self.conv_ones, None, self.conv_w, self.conv_b, window, ctx.seq_of, ctx.cu_seqlens, ctx.slots, x,
                     weight_t=self.conv_w_t)
        # the window is next read by the next step: its update leaves the chain (joined before this mixer returns)
        here = torch.cuda.current_stream(x.device)
        update = branches.branch_stream(x.device, "window")
        with branches.fork(here, update):
            K.conv1d_window_update(raw_x, self.conv_ones, None, window, ctx.cu_seqlens, ctx.slots, ctx.n_seq, self.taps)
        streaming.linear(x, self.w_x, low, ctx)
        raw_dt = ws.alloc((T, I), proj.dtype)
        streaming.linear(low[:, :self.rank_padded], self.w_dt, raw_dt, ctx)
        plan = K.selective_scan_plan(ctx.new_lens, I, self.d_state, proj.dtype)
        scratch = None
        if plan[1] > ctx.n_seq:
            scratch = ws.alloc((plan[1] * I * (self.d_state + 1),), torch.float32)
        K.selective_scan(x, raw_dt, low, self.off_b, self.off_c, z, self.dt_bias, self.a_log, self.d_skip, state,
                         ctx.cu_seqlens, ctx.slots, ctx.n_seq, plan, scratch, y)
        here.wait_stream(update)
        return y


register_mixer("mamba1", SelectiveScanMixer)
