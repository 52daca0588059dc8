"""Nikodra as a ModelSpec.

    x = embed[token] + bigram[row(previous token, token)]
    per layer:  x <- x + m post(mixer(norm(x)));  x <- x + m post(ffn(norm(x)))       (where the layer has a feed-forward)
    logits = head . norm(x)

m is one constant; every norm on the stream is an RMS norm over the whole row with its weight stored around zero.
Mixers: grouped-query attention with biased projections, normed queries and keys, scaled rotary frequencies and values
mixed with those of the first mixing layer (`parts.head_norm_attention`); chunked attention without positions beside
retention, half the sum of the two, each normed (`parts.parallel`, `parts.recurrent`); time mixing with a decay per
key channel and token (`parts.time_mix`).  Both softmaxes hold a one besides the exponentials of the scores.
Feed-forward: one matrix, the exact GELU, one matrix.

Tensor names: embed, bigram, head, final.norm; per layer l<i>.norm1, norm1b, norm2, norm2b, l<i>.mix.*, l<i>.mlp.*.
"""
from __future__ import annotations

from ..config.nikodra import NikodraConfig, NikodraLayerConfig
from ..parts.base import LayerCall, ModelSpec, PartSpec
from ..parts.block import prenorm_layer

# constants of the design
BRANCH_SCALE = 0.5       # the parallel mixer is half the sum of its two normed branches
CARRIED_VALUES = "v_first"   # what the first mixing layer leaves for the later ones of the same step


def _norm(name: str, cfg: NikodraConfig, multiplier: float = 1.0) -> PartSpec:
    return PartSpec("rmsnorm", name, {"eps": cfg.norm_eps, "offset": 1.0, "tensor": "", "multiplier": multiplier})


def _mixer(cfg: NikodraConfig, i: int, layer: NikodraLayerConfig) -> PartSpec:
    if layer.attention is not None:
        m = layer.attention
        mixing = {}
        if m.v_mix:
            mixing = {"value_mix": "first" if i == cfg.first_mixing_layer() else "later", "carried_values": CARRIED_VALUES}
        return PartSpec("head_norm_attention", "mix", {
            "heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "bias": True,
            "qk_norm": "weight", "norm_eps": cfg.norm_eps, "rot_dims": m.rot_dims, "rot_base": m.rot_base,
            "rot_layout": "pairs", "rot_yarn": m.rot_scaling, "one_more": True, **mixing})
    if layer.wkv is not None:
        m = layer.wkv
        return PartSpec("time_mix", "mix", {"heads": m.heads, "dim": m.dim, "decay_rank": m.decay_rank, "norm_eps": cfg.norm_eps})
    left, right = layer.left, layer.right
    return PartSpec("normed_parallel", "mix", {"eps": cfg.norm_eps, "scale": BRANCH_SCALE, "branches": [
        {"name": "left", "kind": "head_norm_attention", "params": {
            "heads": left.heads, "kv_heads": left.kv_heads, "dim": left.dim, "vdim": left.vdim, "scale": left.scale,
            "bias": False, "qk_norm": "unit", "norm_eps": cfg.norm_eps, "chunk": left.chunk, "one_more": True}},
        {"name": "right", "kind": "retention", "params": {
            "heads": right.heads, "dim": right.dim, "vdim": right.vdim, "decay": tuple(right.decay), "norm_eps": cfg.norm_eps,
            "rot_dims": right.rot_dims, "rot_base": right.rot_base}},
    ]})


def model_spec(cfg: NikodraConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(cfg.layers):
        ffn = ffn_norm = ffn_post = None
        if layer.ff is not None:
            ffn = PartSpec("mlp", "mlp", {"intermediate_size": layer.ff, "activation": "gelu", "tensors": ("up", "down")})
            ffn_norm, ffn_post = _norm("norm2", cfg), _norm("norm2b", cfg, cfg.residual_mult)
        layers.append(prenorm_layer(f"l{i}.", _norm("norm1", cfg), (_mixer(cfg, i, layer),), ffn_norm, ffn,
                                    mixer_post_norm=_norm("norm1b", cfg, cfg.residual_mult), ffn_post_norm=ffn_post))
    bigram = None
    if cfg.bigram is not None:
        b = cfg.bigram
        bigram = PartSpec("bigram", "bigram", {"buckets": b.buckets, "mul_prev": b.mul_prev, "mul_cur": b.mul_cur})
    return ModelSpec(
        hidden_size=cfg.hidden_size,
        vocab_size=cfg.vocab_size,
        embedding_name="embed",
        embedding_multiplier=1.0,
        layers=tuple(layers),
        order=tuple(LayerCall(i, i) for i in range(len(layers))),
        final_norm=_norm("final.norm", cfg),
        head_name="head",
        head_multiplier=1.0,
        eos_token_id=-1,
        bos_token_id=0,
        embedding_addend=bigram,
    )
