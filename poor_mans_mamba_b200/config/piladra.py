"""Typed configuration of the Piladra architecture, read from its own config.json keys.

    architecture: "Piladra"; vocab, width; norm: {eps, groups}; canon: {taps}; residual_mult;
    logit_softcap (may be absent or null: none);
    loop (may be absent or null): {start, stop, times};
    layers: [{type, mixer, mlp}], type "attention", "latent_attention" or "mamba1";
      "attention" mixer: {heads, kv_heads, dim, vdim, scale, mask: {size},
                          rot: {dims, base, scaling: {factor, low, high, original}}};
      "latent_attention" mixer: {heads, dim, rot_dim, vdim, kv_rank, scale, rot: {dims, base}};
      "mamba1" mixer: {inner, state, dt_rank, conv};
      mlp: null, {kind: "dense", ff} or
           {kind: "moe", router: {experts, top}, expert: {ff}, shared: {ff} (may be absent or null)}.

Every size and constant comes from the file.  ``mask`` (or its ``size``) may be absent: every earlier token
is seen; ``rot`` and ``rot.scaling`` may be absent (no rotation, frequencies as they are).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, KeyReader
from .boketar import _positive, _sub
from .gikovik import LoopConfig
from .sorovik import _float, _mask, _rotation

LAYER_TYPES = ("attention", "latent_attention", "mamba1")


@dataclass(frozen=True)
class PiladraAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int
    rot_base: float
    rot_scaling: Optional[Tuple[float, float, float, float]]  # factor, low, high, original
    window: int       # 0: every earlier token


@dataclass(frozen=True)
class PiladraLatentConfig:
    heads: int
    dim: int          # unrotated query/key entries per head
    rot_dim: int      # rotated entries per head (one key part shared by all heads)
    vdim: int
    kv_rank: int
    scale: float
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class PiladraScanConfig:
    inner: int
    state: int
    dt_rank: int
    conv: int


@dataclass(frozen=True)
class PiladraDenseConfig:
    ff: int


@dataclass(frozen=True)
class PiladraRoutedConfig:
    experts: int
    top: int
    expert_ff: int
    shared_ff: int    # 0: no shared expert


@dataclass(frozen=True)
class PiladraLayerConfig:
    type: str
    attention: Optional[PiladraAttentionConfig]
    latent: Optional[PiladraLatentConfig]
    scan: Optional[PiladraScanConfig]
    dense: Optional[PiladraDenseConfig]
    routed: Optional[PiladraRoutedConfig]


@dataclass(frozen=True)
class PiladraConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    norm_groups: int
    canon_taps: int
    residual_mult: float
    logit_softcap: float   # 0: none
    layers: Tuple[PiladraLayerConfig, ...]
    loop: Optional[LoopConfig]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """[(layer, the number of the pass of the loop that starts with it, or None)] in the order the layers run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        lp = self.loop
        out: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(lp.start)]
        for t in range(lp.times):
            out += [(i, t if i == lp.start else None) for i in range(lp.start, lp.stop)]
        return out + [(i, None) for i in range(lp.stop, n)]

    @staticmethod
    def from_dict(data: Dict[str, Any]) -> "PiladraConfig":
        top = KeyReader(data)
        vocab, width = _positive(top, "vocab", ""), _positive(top, "width", "")
        norm = KeyReader(_sub(data, "norm", ""))
        eps, groups = _float(norm, "eps", "norm."), _positive(norm, "groups", "norm.")
        if width % groups:
            raise ConfigError(f"config field 'norm.groups': {groups} does not divide the width {width}")
        taps = _positive(KeyReader(_sub(data, "canon", "")), "taps", "canon.")
        cap = top.float("logit_softcap", 0.0)
        if cap < 0.0:
            raise ConfigError(f"config field 'logit_softcap': must not be negative, got {cap}")
        raw_layers = data.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config field 'layers': expected a non-empty list")
        layers = tuple(_layer(entry, i) for i, entry in enumerate(raw_layers))
        loop = None
        if data.get("loop") is not None:
            r = KeyReader(_sub(data, "loop", ""))
            start, stop, times = r.int("start"), r.int("stop"), _positive(r, "times", "loop.")
            if not 0 <= start < stop <= len(layers):
                raise ConfigError(f"config field 'loop': start {start} and stop {stop} must name a span of the {len(layers)} layers")
            loop = LoopConfig(start, stop, times)
        return PiladraConfig(vocab, width, eps, groups, taps, top.float("residual_mult"), cap, layers, loop)


def _layer(entry: Any, i: int) -> PiladraLayerConfig:
    where = f"layers[{i}]."
    if not isinstance(entry, dict):
        raise ConfigError(f"config field 'layers[{i}]': expected an object")
    kind = KeyReader(entry).str("type")
    if kind not in LAYER_TYPES:
        raise ConfigError(f"config field '{where}type': unknown layer type '{kind}' (known: {', '.join(LAYER_TYPES)})")
    mixer, at = _sub(entry, "mixer", where), where + "mixer."
    dense = routed = None
    if entry.get("mlp") is not None:
        mlp = _sub(entry, "mlp", where)
        mkind = KeyReader(mlp).str("kind")
        if mkind == "dense":
            dense = PiladraDenseConfig(_positive(KeyReader(mlp), "ff", where + "mlp."))
        elif mkind == "moe":
            routed = _routed(mlp, where + "mlp.")
        else:
            raise ConfigError(f"config field '{where}mlp.kind': unknown feed-forward '{mkind}' (known: dense, moe)")
    return PiladraLayerConfig(
        kind, _attention(mixer, at) if kind == "attention" else None,
        _latent(mixer, at) if kind == "latent_attention" else None, _scan(mixer, at) if kind == "mamba1" else None,
        dense, routed)


def _attention(mixer: Dict[str, Any], where: str) -> PiladraAttentionConfig:
    r = KeyReader(mixer)
    heads, kv_heads = _positive(r, "heads", where), _positive(r, "kv_heads", where)
    dim, vdim = _positive(r, "dim", where), _positive(r, "vdim", where)
    if heads % kv_heads:
        raise ConfigError(f"config field '{where}kv_heads': {kv_heads} does not divide the {heads} heads")
    rot_dims, base = _rotation(mixer, where, dim)
    scaling = None
    if (mixer.get("rot") or {}).get("scaling") is not None:
        at = where + "rot.scaling."
        s = KeyReader(_sub(mixer["rot"], "scaling", where + "rot."))
        scaling = tuple(_float(s, k, at) for k in ("factor", "low", "high", "original"))
        if scaling[0] <= 0.0 or scaling[3] <= 0.0 or scaling[1] > scaling[2]:
            raise ConfigError(f"config field '{where}rot.scaling': factor and original must be positive and low at most high")
    window, _ = _mask(mixer, where)
    return PiladraAttentionConfig(heads, kv_heads, dim, vdim, _float(r, "scale", where), rot_dims, base, scaling, window)


def _latent(mixer: Dict[str, Any], where: str) -> PiladraLatentConfig:
    r = KeyReader(mixer)
    heads, dim, vdim = _positive(r, "heads", where), _positive(r, "dim", where), _positive(r, "vdim", where)
    kv_rank = _positive(r, "kv_rank", where)
    rot_dim = r.int("rot_dim", 0)
    if rot_dim < 0:
        raise ConfigError(f"config field '{where}rot_dim': must not be negative, got {rot_dim}")
    rot_dims, base = _rotation(mixer, where, rot_dim)
    return PiladraLatentConfig(heads, dim, rot_dim, vdim, kv_rank, _float(r, "scale", where), rot_dims, base)


def _scan(mixer: Dict[str, Any], where: str) -> PiladraScanConfig:
    r = KeyReader(mixer)
    return PiladraScanConfig(*(_positive(r, k, where) for k in ("inner", "state", "dt_rank", "conv")))


def _routed(mlp: Dict[str, Any], where: str) -> PiladraRoutedConfig:
    router = KeyReader(_sub(mlp, "router", where))
    experts, top = _positive(router, "experts", where + "router."), _positive(router, "top", where + "router.")
    if top > experts:
        raise ConfigError(f"config field '{where}router.top': {top} is more than the {experts} experts")
    expert_ff = _positive(KeyReader(_sub(mlp, "expert", where)), "ff", where + "expert.")
    shared_ff = 0
    if mlp.get("shared") is not None:
        shared_ff = _positive(KeyReader(_sub(mlp, "shared", where)), "ff", where + "shared.")
    return PiladraRoutedConfig(experts, top, expert_ff, shared_ff)
