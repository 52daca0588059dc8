"""Norms with the residual additions folded in: RMSNorm and the statistic-free tanh norm.

The RMS norm may take its root mean square over ``groups`` equal neighbouring parts of the row instead of
the whole row (`Norm.group_prologue`; the fold, a vector that waits on the stream and the convolution of a
sublayer's input then share its launch, csrc/fold_norm.cu).

y = x * (1/sqrt(mean(x^2) + eps)) * w; eps inside the root, the weight multiplies after
normalisation (reference src/ops/cpu/rms_norm.cpp:11-16).  Statistics are float32.  A weight
stored around zero (y = ... * (1 + w)) is the same norm with ``offset`` 1.  The RMS norm also serves as
the *post* norm of a sublayer's result, x <- x + rms(result) * w: the launch that norms the next
sublayer's input does both (`folds_post`).
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops as K
from .base import Norm, ParamSpec, register_norm

Tensor = torch.Tensor


def fold_branches(h: Tensor, pending) -> None:
    """h <- h + sum(scale_i * branch_i), two branches per launch."""
    items = list(pending)
    while items:
        K.add_rmsnorm(h, items[:2], None, 0.0, None)
        items = items[2:]


class RMSNorm(Norm):
    """``offset``: the stored weight is kept around zero and the norm multiplies by offset + w (the sum
    is made once, in float32, when the tensors are bound).  ``multiplier``: a constant that the weight takes in (as a
    post norm: the factor with which the normed result joins the stream).  ``tensor``: the weight's name within the
    part ("" where the part's own name is the tensor's).  ``groups``: the row is cut into that many equal
    neighbouring parts and each is divided by its own root mean square."""

    def __init__(self, width: int, eps: float, offset: float = 0.0, tensor: str = "weight", groups: int = 1,
                 multiplier: float = 1.0):
        if groups < 1 or width % groups:
            raise ValueError("the norm's groups must divide the width")
        self.groups = int(groups)
        self.width = int(width)
        self.eps = float(eps)
        self.offset = float(offset)
        self.multiplier = float(multiplier)
        self.tensor = str(tensor)
        self.weight: Optional[Tensor] = None

    def param_specs(self) -> List[ParamSpec]:
        init = ("ones",) if self.offset == 0.0 else ("normal", 0.1)
        return [ParamSpec(self.tensor, (self.width,), kind="vector", init=init)]

    def bind(self, params: Dict[str, Tensor]) -> None:
        w = params[self.tensor]
        if self.offset != 0.0:
            w = w + self.offset
        if self.multiplier != 1.0:
            w = w * self.multiplier
        self.weight = w.contiguous()

    def rms_prologue(self):
        return (self.weight, self.eps) if self.groups == 1 else None

    def group_prologue(self):
        return self.weight, self.eps, self.groups

    def folds_post(self, post: Norm) -> bool:
        return isinstance(post, RMSNorm) and self.groups == 1 and post.groups == 1

    def folds_post_bias(self) -> bool:
        return self.groups == 1

    def forward(self, h: Tensor, pending, out: Tensor, rows: Optional[Tensor], ctx, post: Optional[Norm] = None,
                post_bias: Optional[Tensor] = None) -> None:
        items = list(pending)
        if post is not None and items:
            # a sublayer's result, normed once more before it joins: x <- x + post(sum), out = norm(x), one launch
            if not self.folds_post(post) or len(items) > 2:
                raise ValueError("the RMS norm folds a post norm of its own kind over at most two branches")
            K.add_postnorm_rmsnorm(h, items, post.weight, post.eps, self.weight, self.eps, out, rows, bias=post_bias)
            return
        while len(items) > 2:  # more than two branches: fold the surplus first
            if rows is not None:
                raise ValueError("row-selected norm takes at most two pending branches")
            K.add_rmsnorm(h, items[:2], None, 0.0, None)
            items = items[2:]
        if self.groups > 1:
            K.fold_norm(h, h, items, None, self.weight, self.eps, self.groups, out, rows)
        else:
            K.add_rmsnorm(h, items, self.weight, self.eps, out, rows)

    def _whole_row(self) -> None:
        if self.groups > 1:
            raise NotImplementedError("an RMS norm over groups of channels cannot norm a sublayer's result")

    def apply(self, pending, out: Tensor, ctx, post_bias: Optional[Tensor] = None) -> None:
        self._whole_row()
        K.add_postnorm_rmsnorm(None, list(pending), self.weight, self.eps, None, 0.0, out, bias=post_bias)

    def fold(self, h: Tensor, pending, ctx, post_bias: Optional[Tensor] = None) -> None:
        self._whole_row()
        K.add_postnorm_rmsnorm(h, list(pending), self.weight, self.eps, None, 0.0, None, bias=post_bias)


class TanhNorm(Norm):
    """y = tanh(alpha * x) * w + b: a scalar ``alpha``, vectors w and b; no mean, no variance, no eps.
    Tensors: ``tensor`` (the weight; "" where the part's own name is the tensor's), ``b``, ``alpha``
    (a tensor of one value).  Being element-wise it serves before a sublayer as well as after one:
    as the post norm of a sublayer's result it is folded into the launch that norms the next
    sublayer's input (`folds_post`)."""

    def __init__(self, width: int, tensor: str = "weight", bias: str = "b", alpha: str = "alpha",
                 alpha_init: float = 1.0):
        self.width = int(width)
        self.tensor, self.bias_name, self.alpha_name = str(tensor), str(bias), str(alpha)
        self.alpha_init = float(alpha_init)
        self.trio = None

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec(self.tensor, (self.width,), kind="vector", init=("uniform", 0.5, 1.5)),
                ParamSpec(self.bias_name, (self.width,), kind="vector", init=("normal", 0.1)),
                ParamSpec(self.alpha_name, (), kind="vector", init=("uniform", 0.5 * self.alpha_init, 1.5 * self.alpha_init))]

    def bind(self, params: Dict[str, Tensor]) -> None:
        self.trio = (params[self.alpha_name].reshape(1).contiguous(), params[self.tensor].contiguous(),
                     params[self.bias_name].contiguous())

    def folds_post(self, post: Norm) -> bool:
        return isinstance(post, TanhNorm)

    def forward(self, h: Tensor, pending, out: Tensor, rows: Optional[Tensor], ctx, post: Optional[Norm] = None) -> None:
        items = list(pending)
        if len(items) > 2:
            raise ValueError("the tanh norm folds at most two pending branches")
        if post is not None and not isinstance(post, TanhNorm):
            raise ValueError("the tanh norm folds a post norm of its own kind only")
        K.add_tanh_norm(h, items, post.trio if post is not None and items else None, self.trio, out, rows)

    def apply(self, pending, out: Tensor, ctx) -> None:
        K.add_tanh_norm(None, list(pending), None, self.trio, out, None)

    def fold(self, h: Tensor, pending, ctx) -> None:
        K.add_tanh_norm(h, list(pending), self.trio, None, None, None)


register_norm("rmsnorm", RMSNorm)
register_norm("tanh_norm", TanhNorm)
