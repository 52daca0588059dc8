"""Piladra as a ModelSpec.

    x = embed[token]
    per layer:  x <- x + m mixer(c(norm(x)));  x <- x + m ffn(c(norm(x)))       (where the layer has a feed-forward)
    logits = cap tanh(head . norm(x) / cap)

m is one constant; every norm is an RMS norm over groups of channels with a plain weight; c adds a short causal
convolution over time to its input (`parts.input_conv`), with state of its own in every layer and for either
sublayer.  Mixers: grouped-query attention with scaled rotary frequencies, normed values, a sliding window and a
sink per head (`parts.gated_attention`); latent attention with queries straight from its input, one rotated key
part shared by all heads and a gate per channel (`parts.latent_attention`); Mamba-1 (`parts.selective_scan`).
Feed-forward: dense SwiGLU, or experts chosen by their sigmoid scores, whose scores multiply their inputs, beside a
shared expert (`parts.moe`).  A span of layers may run several times in a row with the same tensors, every run on a
cache of its own; before every pass the pass's vector joins the stream (`parts.stream_update.PassStep`).

Tensor names: embed, head, final.norm, loop.step; per layer l<i>.norm1, norm2, canon1, canon2, l<i>.mix.*, l<i>.mlp.*.
"""
from __future__ import annotations

import math

from ..config.piladra import PiladraConfig, PiladraLayerConfig
from ..parts.base import LayerCall, ModelSpec, PartSpec
from ..parts.block import prenorm_layer

_DENSE_TENSORS = ("gate", "up", "down")


def _norm(name: str, cfg: PiladraConfig) -> PartSpec:
    return PartSpec("rmsnorm", name, {"eps": cfg.norm_eps, "groups": cfg.norm_groups, "tensor": ""})


def _input(name: str, cfg: PiladraConfig) -> PartSpec:
    return PartSpec("residual_conv", name, {"taps": cfg.canon_taps})


def _mixer(cfg: PiladraConfig, layer: PiladraLayerConfig) -> PartSpec:
    if layer.attention is not None:
        m = layer.attention
        return PartSpec("rotary_gated_attention", "mix", {
            "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "rot_dims": m.rot_dims,
            "rot_base": m.rot_base, "rot_scaling": m.rot_scaling, "rot_layout": "halves", "scale": m.scale, "bias": False,
            "gate": False, "window": m.window, "sink": True, "value_norm_eps": cfg.norm_eps,
            "out_multiplier": cfg.residual_mult})
    if layer.latent is not None:
        m = layer.latent
        return PartSpec("latent_attention", "mix", {
            "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "q_rank": 0, "kv_rank": m.kv_rank, "scale": m.scale,
            "norm_eps": cfg.norm_eps, "rot_dim": m.rot_dim, "rot_dims": m.rot_dims, "rot_base": m.rot_base,
            "rot_layout": "halves", "sink": False, "gate": "channel", "out_multiplier": cfg.residual_mult})
    m = layer.scan
    return PartSpec("mamba1", "mix", {"inner": m.inner, "state": m.state, "dt_rank": m.dt_rank, "conv": m.conv,
                                      "out_multiplier": cfg.residual_mult})


def _feed_forward(cfg: PiladraConfig, layer: PiladraLayerConfig):
    if layer.dense is not None:
        return PartSpec("swiglu", "mlp", {"intermediate_size": layer.dense.ff, "tensors": _DENSE_TENSORS,
                                          "down_multiplier": cfg.residual_mult})
    if layer.routed is not None:
        r = layer.routed
        # the experts' activation silu(g) * u is the clamped gated form without a limit, slope 1 and no shift
        return PartSpec("routed_glu", "mlp", {
            "experts": r.experts, "top": r.top, "expert_ff": r.expert_ff, "expert_limit": math.inf,
            "shared_ff": r.shared_ff, "shared_limit": math.inf, "act_alpha": 1.0, "act_shift": 0.0, "router_bias": False,
            "router": "sigmoid", "weigh": "input", "out_multiplier": cfg.residual_mult})
    return None


def model_spec(cfg: PiladraConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(cfg.layers):
        ffn = _feed_forward(cfg, layer)
        has = ffn is not None
        layers.append(prenorm_layer(
            f"l{i}.", _norm("norm1", cfg), (_mixer(cfg, layer),), _norm("norm2", cfg) if has else None, ffn,
            mixer_input=_input("canon1", cfg), ffn_input=_input("canon2", cfg) if has else None))
    # every run of a layer has a cache of its own: cache ids count the runs
    order = tuple(LayerCall(layer, run, begins is not None, begins or 0) for run, (layer, begins) in enumerate(cfg.runs()))
    return ModelSpec(
        hidden_size=cfg.hidden_size,
        vocab_size=cfg.vocab_size,
        embedding_name="embed",
        embedding_multiplier=1.0,
        layers=tuple(layers),
        order=order,
        final_norm=_norm("final.norm", cfg),
        head_name="head",
        head_multiplier=1.0,
        eos_token_id=-1,
        bos_token_id=0,
        reentry=PartSpec("pass_step", "loop", {"passes": cfg.loop.times}) if cfg.loop is not None else None,
        logit_softcap=cfg.logit_softcap,
    )
