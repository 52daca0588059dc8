"""Softmax attention with a norm per query and key head, and options that belong to it.

    q = Wq x + bq (heads x dim), k = Wk x + bk (kv_heads x dim), v = Wv x + bv (kv_heads x vdim) (``bias``);
    ``qk_norm``: every query and key head is divided by its own root mean square over dim (eps inside the root),
    with "weight" then multiplied by a weight of size dim that all heads share; None: left as it is;
    then the first rot_dims entries of every q and k head turn in pairs, entries (2i, 2i+1) (``rot_layout`` "pairs")
    or (i, i + rot_dims/2) ("halves"), by the angle p * f_i, f_i = rot_base^(-2i / rot_dims); ``rot_yarn`` (factor,
    original, fast, slow): frequencies and amplitude of `parts.rope.yarn_frequencies`; rot_dims 0: no positions;
    ``value_mix``: v <- (1 - l) v + l v0 with l the scalar tensor ``vmix`` and v0 the values that the layer with
    "first" left for the same tokens in the step's carried rows (``carried_values``); layers with "later" take them;
    score = (q . k) * scale; token i sees every j <= i, with ``chunk`` only those of its own chunk of that many
    positions (counted from position 0), with ``window`` only 0 <= i - j < window;
    p_j = exp(s_j) / (one_more + sum exp(s_j)) with ``one_more`` 1 (a sink whose score is 0) or 0;
    out = Wo [heads] (+ bo with ``bias``).

Query head h reads key/value head h // (heads / kv_heads).  State per request: the normed, rotated keys and the (mixed)
values in cache pages.  Biases, norms, rotation, mixing and the page write are one launch (a warp per head); heads
are padded with zeros to Dp = max(dim, vdim) rounded up to a multiple of 16 there and in the attention kernels.
Norms, positions, angles, scores and softmax weights are float arithmetic in both storage types.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from ..kernels import ops as K
from . import streaming
from .base import ParamSpec, StateSpec, register_mixer
from .rope import rotary_frequencies, yarn_frequencies
from .window_attention import PagedSoftmaxAttention

Tensor = torch.Tensor


class HeadNormAttention(PagedSoftmaxAttention):
    def __init__(self, hidden_size: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, norm_eps: float,
                 bias: bool = False, qk_norm: Optional[str] = "unit", rot_dims: int = 0, rot_base: float = 1.0,
                 rot_layout: str = "pairs", rot_yarn: Optional[Sequence[float]] = None, window: int = 0, chunk: int = 0,
                 one_more: bool = False, value_mix: Optional[str] = None, carried_values: str = "values",
                 out_multiplier: float = 1.0):
        if heads % kv_heads:
            raise ValueError("query heads must be a multiple of key/value heads")
        if rot_dims % 2 or not 0 <= rot_dims <= dim:
            raise ValueError("rot_dims must be even and at most dim")
        if rot_layout not in ("halves", "pairs"):
            raise ValueError("rot_layout is 'halves' or 'pairs'")
        if qk_norm not in (None, "unit", "weight"):
            raise ValueError("qk_norm is None, 'unit' or 'weight'")
        if value_mix not in (None, "first", "later"):
            raise ValueError("value_mix is None, 'first' or 'later'")
        if window < 0 or chunk < 0 or (window > 0 and chunk > 0):
            raise ValueError("a window or chunks, neither negative")
        self.hidden_size = int(hidden_size)
        self.heads, self.kv_heads, self.dim, self.vdim = int(heads), int(kv_heads), int(dim), int(vdim)
        self.scale, self.norm_eps = float(scale), float(norm_eps)
        self.has_bias, self.qk_norm, self.one_more = bool(bias), qk_norm, bool(one_more)
        self.rot_dims, self.rot_base, self.half_layout = int(rot_dims), float(rot_base), rot_layout == "halves"
        self.rot_yarn = None if rot_yarn is None else tuple(float(v) for v in rot_yarn)
        self.window, self.chunk = int(window), int(chunk)
        self.value_mix, self.carried_values = value_mix, str(carried_values)
        self.out_scale = float(out_multiplier)
        self.padded_dim = (max(self.dim, self.vdim) + 15) // 16 * 16
        K.check_head_dim(self.padded_dim)
        self.q_dim, self.k_dim, self.v_dim = self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim
        self.inv_freq: Optional[Tensor] = None
        self.amplitude = 1.0
        self.biases = self.out_bias = self.norm_weights = self.mix_weight = self.sink = None

    def param_specs(self) -> List[ParamSpec]:
        D = self.hidden_size
        specs = []
        for name, rows in (("q", self.q_dim), ("k", self.k_dim), ("v", self.v_dim)):
            specs.append(ParamSpec(name, (rows, D)))
            if self.has_bias:
                specs.append(ParamSpec(name + ".b", (rows,), kind="vector", init=("normal", 0.1)))
        if self.qk_norm == "weight":
            specs += [ParamSpec(name + ".norm", (self.dim,), kind="vector", init=("uniform", 0.5, 1.5)) for name in ("q", "k")]
        if self.value_mix == "later":
            specs.append(ParamSpec("vmix", (), kind="vector", init=("uniform", 0.2, 0.8)))
        specs.append(ParamSpec("o", (D, self.heads * self.vdim)))
        if self.has_bias:
            specs.append(ParamSpec("o.b", (D,), kind="vector", init=("normal", 0.1)))
        return specs

    def ignored_names(self) -> List[str]:
        return ["vmix"] if self.value_mix == "first" else []  # a checkpoint may hold the weight of a layer that has nothing to mix

    def carries(self) -> Dict[str, int]:
        return {self.carried_values: self.v_dim} if self.value_mix is not None else {}

    def state_specs(self) -> List[StateSpec]:
        return [StateSpec.paged("kv", planes=2, width=self.kv_heads * self.padded_dim, window=self.window, chunk=self.chunk)]

    def bind(self, params: Dict[str, Tensor]) -> None:
        self.w_in = torch.cat([params["q"], params["k"], params["v"]], dim=0).contiguous()
        if self.has_bias:
            self.biases = tuple(params[n + ".b"].contiguous() for n in ("q", "k", "v"))
            self.out_bias = params["o.b"].contiguous()
        if self.qk_norm == "weight":
            self.norm_weights = (params["q.norm"].contiguous(), params["k.norm"].contiguous())
        if self.value_mix == "later":
            self.mix_weight = params["vmix"].reshape(1).contiguous()
        w_o = params["o"]
        if self.one_more:  # a sink per head whose score is 0
            self.sink = torch.zeros(self.heads, dtype=torch.float32, device=w_o.device)
        if self.padded_dim != self.vdim:  # zero columns where the attention kernel's heads are padded
            w = torch.zeros((w_o.shape[0], self.heads, self.padded_dim), dtype=w_o.dtype, device=w_o.device)
            w[:, :, :self.vdim] = w_o.view(w_o.shape[0], self.heads, self.vdim)
            w_o = w.view(w_o.shape[0], self.heads * self.padded_dim)
        self.w_out = w_o.contiguous()

    def finalize(self, dtype: torch.dtype, device: torch.device) -> None:
        if self.rot_dims > 0:
            if self.rot_yarn is not None:
                f, self.amplitude = yarn_frequencies(self.rot_dims, self.rot_base, *self.rot_yarn)
            else:
                f = rotary_frequencies(self.rot_dims, self.rot_base)
            self.inv_freq = f.to(device).contiguous()
        self._make_split_counter(device)

    def output_weight(self) -> Tensor:
        return self.w_out

    def output_bias(self) -> Optional[Tensor]:
        return self.out_bias

    def forward_projected(self, proj: Tensor, ctx, cache, out: Tensor) -> None:
        streaming.linear(self.pre_output(proj, ctx, cache), self.w_out, out, ctx)
        if self.out_bias is not None and not ctx.defer_output_bias:
            K.add_row_bias_(out, self.out_bias)

    def pre_output(self, proj: Tensor, ctx, cache) -> Tensor:
        """The concatenated (padded) heads [T, heads * Dp]."""
        T = proj.shape[0]
        ws = ctx.workspace
        kv = cache.paged(f"{self.name}.kv")
        H, G, Dp = self.heads, self.kv_heads, self.padded_dim
        c_k, c_v = self.q_dim, self.q_dim + self.k_dim
        values = ctx.carried[self.carried_values] if self.value_mix is not None else None
        q_rot = ws.alloc((T, H * Dp), proj.dtype)
        K.head_norm_rope_store(proj[:, :c_k], proj[:, c_k:c_v], proj[:, c_v:c_v + self.v_dim], self.inv_freq, self.rot_dims,
                               ctx.positions, ctx.seq_of, kv.block_table, kv.pool, q_rot, H, G, self.dim, self.vdim, Dp,
                               half_layout=self.half_layout, amplitude=self.amplitude, biases=self.biases,
                               norm_eps=self.norm_eps if self.qk_norm is not None else None, norm_weights=self.norm_weights,
                               values=values, mix_weight=self.mix_weight)
        attn = ws.alloc((T, H * Dp), proj.dtype)
        self._attend(q_rot, kv, ctx, attn)
        return attn


register_mixer("head_norm_attention", HeadNormAttention)
