"""Time mixing: linear attention whose inputs look one token back, with a decay per key channel and token.

    with h' the token before h (zeros before the sequence's start), every one of r, k, v, g, w reads its own mix
    h + (h' - h) mu_s;  r, k, v = W_s mix_s (heads x dim);  gate = silu(W_g mix_g);
    decay w = exp(-exp(W_w2 tanh(W_w1 mix_w) + w0)) per head and key channel;
    per head, from a zero state:  o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T;
    out = Wo [ (o / sqrt(mean(o^2) + eps) per head) * norm * gate ].

State per request (float32, in slots): the last token's h [D] and S [heads, dim, dim].  The decays (from W_w2's float
sums on), the recurrence, the norm and the gate are float arithmetic in both storage types; projections and mixes have
the storage type.  The five mixes are one launch; steps of few tokens run the five products that read them as one
weight-streaming launch, longer steps the four of equal size as one batched product.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..kernels import ops as K
from . import branches, streaming
from .base import Mixer, ParamSpec, StateSpec, register_mixer
from .recurrent import run_recurrence

Tensor = torch.Tensor

_STREAMS = ("r", "k", "v", "g", "w")   # the order of the mixes; the first four share one stacked weight


class TimeMix(Mixer):
    def __init__(self, hidden_size: int, heads: int, dim: int, decay_rank: int, norm_eps: float, out_multiplier: float = 1.0):
        if dim > K.RECURRENT_MAX_KEY_DIM:
            raise ValueError(f"the recurrence kernels take key sizes up to {K.RECURRENT_MAX_KEY_DIM}, got {dim}")
        self.hidden_size, self.heads, self.dim = int(hidden_size), int(heads), int(dim)
        self.decay_rank, self.norm_eps = int(decay_rank), float(norm_eps)
        self.out_scale = float(out_multiplier)
        self.inner = self.heads * self.dim

    def param_specs(self) -> List[ParamSpec]:
        D, I, R = self.hidden_size, self.inner, self.decay_rank
        specs = [ParamSpec(f"mu.{s}", (D,), kind="vector", init=("uniform", 0.0, 1.0)) for s in _STREAMS]
        specs += [ParamSpec(s, (I, D)) for s in _STREAMS[:4]]
        return specs + [ParamSpec("w1", (R, D)), ParamSpec("w2", (I, R)),
                        ParamSpec("w0", (I,), kind="vector", init=("uniform", -4.0, 0.0)),
                        ParamSpec("u", (self.heads, self.dim), kind="vector", init=("normal", 0.5)),
                        ParamSpec("norm", (I,), kind="vector", init=("ones",)), ParamSpec("o", (D, I))]

    def state_specs(self) -> List[StateSpec]:
        return [StateSpec.fixed("h", (self.hidden_size,), "float32"),
                StateSpec.fixed("S", (self.heads, self.dim, self.dim), "float32")]

    def bind(self, params: Dict[str, Tensor]) -> None:
        self.mu = torch.stack([params[f"mu.{s}"] for s in _STREAMS]).contiguous()
        self.w_in = torch.stack([params[s] for s in _STREAMS[:4]]).contiguous()   # [4, inner, D]
        self.w1, self.w2, self.w_out = params["w1"].contiguous(), params["w2"].contiguous(), params["o"].contiguous()
        self.w0, self.bonus = params["w0"].contiguous(), params["u"].reshape(-1).contiguous()
        self.norm_w = params["norm"].contiguous()

    def output_weight(self) -> Tensor:
        return self.w_out

    def streamed_weights(self) -> List[Tensor]:
        return [self.w_in, self.w1, self.w2, self.w_out]

    def forward(self, x: Tensor, ctx, cache, out: Tensor) -> None:
        T, D = x.shape
        I, R, ws = self.inner, self.decay_rank, ctx.workspace
        rows = K.padded_rows(T)
        mixes = ws.alloc((5, rows, D), x.dtype)
        K.shifted_mixes(x, self.mu, cache.fixed(f"{self.name}.h"), ctx.cu_seqlens, ctx.slots, ctx.seq_of, mixes)
        proj = ws.alloc((4, rows, I), x.dtype)
        low = ws.alloc((T, R), x.dtype)
        a = ws.alloc((T, I), torch.float32)
        here = torch.cuda.current_stream(x.device)
        if streaming.linears([mixes[s, :T] for s in range(5)], [*self.w_in, self.w1], [*proj[:, :T], low], ctx):
            K.low_rank_tanh(low, self.w2, a)
            side = None
        else:
            # the low-rank product of the decays beside the four large ones (a parallel branch of a recorded step)
            side = branches.branch_stream(x.device, "gate")
            with branches.fork(here, side):
                K.linear(mixes[4, :T], self.w1, low)
                if T <= K.LOW_RANK_TANH_MAX_TOKENS or x.dtype == torch.float32:
                    K.low_rank_tanh(low, self.w2, a)
                else:
                    K.tanh_(low)
                    K.linear_f32_out(low, self.w2, a, None if K.mm_has_f32_out() else ws.alloc((T, I), x.dtype), 1.0)
            K.batched_linear(mixes[:4], self.w_in, proj)
            here.wait_stream(side)
        o = ws.alloc((T, I), torch.float32)
        run_recurrence("wkv", proj[0, :T], proj[1, :T], proj[2, :T], cache.fixed(f"{self.name}.S"), ctx, o, self.heads, self.dim,
                       self.dim, a=a, a_bias=self.w0, bonus=self.bonus)
        y = ws.alloc((T, I), x.dtype)
        K.gated_norm(o, proj[3, :T], 1.0, None, self.norm_w, self.norm_eps, self.heads, True, y, gate="silu")
        streaming.linear(y, self.w_out, out, ctx)


register_mixer("time_mix", TimeMix)
