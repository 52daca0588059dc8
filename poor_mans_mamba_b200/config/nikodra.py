"""Typed configuration of the Nikodra architecture, read from its own config.json keys.

    architecture: "Nikodra"; vocab, width; norm: {eps}; residual_mult;
    embedding (may be absent or null): {bigram (may be absent or null): {buckets, mul_prev, mul_cur}};
    layers: [{type, mixer, mlp}], type "attention", "parallel" or "wkv";
      "attention" mixer: {heads, kv_heads, dim, vdim, scale, v_mix,
                          rot: {dims, base, scaling: {factor, original, fast, slow}}};
      "parallel" mixer: {left: {heads, kv_heads, dim, vdim, scale, mask: {size}},
                         right: {heads, dim, vdim, decay: [per head], rot: {dims, base}}};
      "wkv" mixer: {heads, dim};
      mlp: null or {kind: "dense", ff}.

Every size and constant comes from the file.  ``mask`` (or its ``size``) may be absent: every earlier token is
seen; ``rot`` and ``rot.scaling`` may be absent (no rotation, frequencies as they are); ``v_mix`` absent is false.
One size is in no key: the inner width of the wkv mixer's low-rank decay (``w1``/``w2``).  It is read from the
shape of ``<layer>.mix.w1`` in the model folder; a configuration without a folder (the random-weights mode) names
it ``decay_rank`` in the mixer's dict.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .base import ConfigError, KeyReader
from .boketar import _heads, _positive, _rank, _sub
from .sorovik import _float, _mask, _rotation

LAYER_TYPES = ("attention", "parallel", "wkv")


@dataclass(frozen=True)
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class NikodraAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int
    rot_base: float
    rot_scaling: Optional[Tuple[float, float, float, float]]  # factor, original, fast, slow
    v_mix: bool


@dataclass(frozen=True)
class NikodraChunkedConfig:
    """The parallel mixer's left side."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int        # 0: every earlier token


@dataclass(frozen=True)
class NikodraRetentionConfig:
    """The parallel mixer's right side."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class NikodraWkvConfig:
    heads: int
    dim: int
    decay_rank: int


@dataclass(frozen=True)
class NikodraLayerConfig:
    type: str
    attention: Optional[NikodraAttentionConfig]
    left: Optional[NikodraChunkedConfig]
    right: Optional[NikodraRetentionConfig]
    wkv: Optional[NikodraWkvConfig]
    ff: Optional[int]   # None: the layer has no feed-forward


@dataclass(frozen=True)
class NikodraConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    residual_mult: float
    bigram: Optional[BigramConfig]
    layers: Tuple[NikodraLayerConfig, ...]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def first_mixing_layer(self) -> Optional[int]:
        """The layer whose values the other layers with ``v_mix`` mix theirs with."""
        return next((i for i, l in enumerate(self.layers) if l.attention is not None and l.attention.v_mix), None)

    @staticmethod
    def from_dict(data: Dict[str, Any], shapes: Optional[Mapping[str, Tuple[int, ...]]] = None) -> "NikodraConfig":
        top = KeyReader(data)
        vocab, width = _positive(top, "vocab", ""), _positive(top, "width", "")
        eps = _float(KeyReader(_sub(data, "norm", "")), "eps", "norm.")
        bigram = None
        if (data.get("embedding") or {}).get("bigram") is not None:
            b, at = KeyReader(_sub(_sub(data, "embedding", ""), "bigram", "embedding.")), "embedding.bigram."
            bigram = BigramConfig(_positive(b, "buckets", at), *(_multiplier(b, k, at) for k in ("mul_prev", "mul_cur")))
        raw_layers = data.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config field 'layers': expected a non-empty list")
        layers = tuple(_layer(entry, i, width, shapes) for i, entry in enumerate(raw_layers))
        cfg = NikodraConfig(vocab, width, eps, top.float("residual_mult"), bigram, layers)
        first = cfg.first_mixing_layer()
        for i, l in enumerate(layers):
            if l.attention is not None and l.attention.v_mix:
                a, b = l.attention, layers[first].attention
                if (a.kv_heads, a.vdim) != (b.kv_heads, b.vdim):
                    raise ConfigError(f"config field 'layers[{i}].mixer.v_mix': its values ({a.kv_heads} heads of {a.vdim}) and "
                                      f"those of layer {first} ({b.kv_heads} of {b.vdim}) differ in size")
        return cfg


def _multiplier(r: KeyReader, key: str, where: str) -> int:
    v = r.int(key)
    if v < 0:
        raise ConfigError(f"config field '{where}{key}': must not be negative, got {v}")
    return v


def _layer(entry: Any, i: int, width: int, shapes) -> NikodraLayerConfig:
    where = f"layers[{i}]."
    if not isinstance(entry, dict):
        raise ConfigError(f"config field 'layers[{i}]': expected an object")
    kind = KeyReader(entry).str("type")
    if kind not in LAYER_TYPES:
        raise ConfigError(f"config field '{where}type': unknown layer type '{kind}' (known: {', '.join(LAYER_TYPES)})")
    mixer, at = _sub(entry, "mixer", where), where + "mixer."
    ff = None
    if entry.get("mlp") is not None:
        mlp = _sub(entry, "mlp", where)
        mkind = KeyReader(mlp).str("kind")
        if mkind != "dense":
            raise ConfigError(f"config field '{where}mlp.kind': unknown feed-forward '{mkind}' (known: dense)")
        ff = _positive(KeyReader(mlp), "ff", where + "mlp.")
    attention = left = right = wkv = None
    if kind == "attention":
        attention = _attention(mixer, at)
    elif kind == "parallel":
        left = _chunked(_sub(mixer, "left", at), at + "left.")
        right = _retention(_sub(mixer, "right", at), at + "right.")
    else:
        r = KeyReader(mixer)
        wkv = NikodraWkvConfig(_positive(r, "heads", at), _positive(r, "dim", at),
                               _rank(mixer, "decay_rank", f"l{i}.mix.w1", width, at, shapes))
    return NikodraLayerConfig(kind, attention, left, right, wkv, ff)


def _attention(mixer: Dict[str, Any], where: str) -> NikodraAttentionConfig:
    r = KeyReader(mixer)
    heads, kv_heads = _heads(r, where)
    dim, vdim = _positive(r, "dim", where), _positive(r, "vdim", where)
    rot_dims, base = _rotation(mixer, where, dim)
    scaling = None
    if (mixer.get("rot") or {}).get("scaling") is not None:
        at = where + "rot.scaling."
        s = KeyReader(_sub(mixer["rot"], "scaling", where + "rot."))
        scaling = tuple(_float(s, k, at) for k in ("factor", "original", "fast", "slow"))
        if min(scaling) <= 0.0:
            raise ConfigError(f"config field '{where}rot.scaling': factor, original, fast and slow must be positive")
        if rot_dims > 0 and base <= 1.0:
            raise ConfigError(f"config field '{where}rot.base': scaled frequencies need a base above 1, got {base}")
    return NikodraAttentionConfig(heads, kv_heads, dim, vdim, _float(r, "scale", where), rot_dims, base, scaling,
                                  r.bool("v_mix", False))


def _chunked(side: Dict[str, Any], where: str) -> NikodraChunkedConfig:
    r = KeyReader(side)
    heads, kv_heads = _heads(r, where)
    chunk, _ = _mask(side, where)
    return NikodraChunkedConfig(heads, kv_heads, _positive(r, "dim", where), _positive(r, "vdim", where),
                                _float(r, "scale", where), chunk)


def _retention(side: Dict[str, Any], where: str) -> NikodraRetentionConfig:
    r = KeyReader(side)
    heads, dim = _positive(r, "heads", where), _positive(r, "dim", where)
    rot_dims, base = _rotation(side, where, dim)
    return NikodraRetentionConfig(heads, dim, _positive(r, "vdim", where), r.float_list("decay", heads), rot_dims, base)
