"""Plain, slow Nikodra forward pass: whole sequences, no cache, one function per mechanism.

The oracle of the Nikodra tests.  It shares no code with the package: the configuration is a plain
dict, the weights a ``name -> tensor`` dict, and every formula runs directly on the CPU in one
floating-point type (float64 by default).  Notation: T tokens, D model width, linear weights stored
[out, in].  Masks are dense T x T tables, rotations act on pairs one by one, recurrences are loops
over tokens with the state as a [key, value] matrix per head.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensor = torch.Tensor


# --------------------------------------------------------------------------- small functions
def linear(x: Tensor, w: Tensor, b: Optional[Tensor] = None) -> Tensor:
    y = x @ w.t()
    return y if b is None else y + b


def silu(z: Tensor) -> Tensor:
    return z * torch.sigmoid(z)


def gelu_erf(z: Tensor) -> Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def rms(x: Tensor, eps: float) -> Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x: Tensor, w: Tensor, eps: float) -> Tensor:
    """The model's norm: the weight is stored around zero."""
    return rms(x, eps) * (1.0 + w)


# --------------------------------------------------------------------------- embedding
def bigram_rows(tokens: List[int], mul_prev: int, mul_cur: int, buckets: int) -> List[int]:
    """Row of the bigram table per token; the first token has no predecessor and takes the row behind the buckets."""
    return [buckets if t == 0 else (tokens[t - 1] * mul_prev + tokens[t] * mul_cur) % buckets for t in range(len(tokens))]


def embed(tokens: List[int], W: Dict[str, Tensor], bigram: Optional[dict]) -> Tensor:
    x = W["embed"][torch.tensor(tokens)]
    if bigram is None:
        return x
    return x + W["bigram"][torch.tensor(bigram_rows(tokens, bigram["mul_prev"], bigram["mul_cur"], bigram["buckets"]))]


# --------------------------------------------------------------------------- positions
def frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> Tensor:
    """f_i = base^(-2i/dims); with ``scaling`` the fast-turning pairs keep theirs, the slow ones are divided by the
    factor, and between the two pair numbers lo and hi (where a pair turns ``fast`` and ``slow`` times within
    ``original`` positions) the two are blended linearly."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is not None:
        def pair_that_turns(times: float) -> float:
            return dims * math.log(scaling["original"] / (2.0 * math.pi * times)) / (2.0 * math.log(base))

        lo = max(math.floor(pair_that_turns(scaling["fast"])), 0)
        hi = min(math.ceil(pair_that_turns(scaling["slow"])), dims - 1)
        for i in range(dims // 2):
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f[i] = f[i] / scaling["factor"] * r + f[i] * (1.0 - r)
    return torch.tensor(f, dtype=torch.float64)


def turn_amplitude(scaling: Optional[dict]) -> float:
    """Factor on the sines and cosines."""
    return 1.0 if scaling is None else 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x: Tensor, positions: Tensor, freq: Tensor, halves: bool, amplitude: float = 1.0) -> Tensor:
    """x [T, heads, d]: pair i is entries (i, i + dims/2) with ``halves``, else (2i, 2i + 1); dims = 2 len(freq)."""
    n = freq.shape[0]
    out = x.clone()
    for i in range(n):
        a, b = (i, i + n) if halves else (2 * i, 2 * i + 1)
        ang = positions.to(torch.float64) * freq[i]
        c, s = (torch.cos(ang) * amplitude).to(x.dtype)[:, None], (torch.sin(ang) * amplitude).to(x.dtype)[:, None]
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


# --------------------------------------------------------------------------- softmax attention
def causal_mask(T: int) -> Tensor:
    return torch.arange(T)[None, :] <= torch.arange(T)[:, None]


def chunk_mask(T: int, size: int) -> Tensor:
    """i sees j <= i of its own chunk of ``size`` positions (0: every j <= i)."""
    if size == 0:
        return causal_mask(T)
    i = torch.arange(T)
    return causal_mask(T) & (i[:, None] // size == i[None, :] // size)


def attend_with_one_more(q: Tensor, k: Tensor, v: Tensor, scale: float, mask: Tensor) -> Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]: query head h reads head h // (H / G); the softmax's denominator holds a
    one besides the exponentials of the visible scores."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        s = ((q[:, h] @ k[:, h // rep].t()) * scale).masked_fill(~mask, -math.inf)
        m = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
        p = torch.exp(s - m)
        out[:, h] = (p / (torch.exp(-m) + p.sum(dim=-1, keepdim=True))) @ v[:, h // rep]
    return out


def attention(x: Tensor, W: Dict[str, Tensor], pre: str, m: dict, eps: float, positions: Tensor, shared: dict) -> Tensor:
    """Biased projections, normed and rotated queries and keys, values mixed with those of the first mixing layer
    (kept in ``shared``), every earlier token visible."""
    T = x.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    freq, amp = frequencies(rot["dims"], rot["base"], rot.get("scaling")), turn_amplitude(rot.get("scaling"))
    q = rms(linear(x, W[pre + "q"], W[pre + "q.b"]).reshape(T, H, d), eps) * W[pre + "q.norm"]
    k = rms(linear(x, W[pre + "k"], W[pre + "k.b"]).reshape(T, G, d), eps) * W[pre + "k.norm"]
    v = linear(x, W[pre + "v"], W[pre + "v.b"]).reshape(T, G, dv)
    if m.get("v_mix"):
        if "v" in shared:
            lam = W[pre + "vmix"]
            v = (1.0 - lam) * v + lam * shared["v"]
        else:
            shared["v"] = v
    q, k = rotate(q, positions, freq, False, amp), rotate(k, positions, freq, False, amp)
    heads = attend_with_one_more(q, k, v, m["scale"], causal_mask(T))
    return linear(heads.reshape(T, H * dv), W[pre + "o"], W[pre + "o.b"])


def chunked_attention(x: Tensor, W: Dict[str, Tensor], pre: str, m: dict, eps: float) -> Tensor:
    """No rotation, unit-rms queries and keys, chunks of mask.size positions."""
    T = x.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(linear(x, W[pre + "q"]).reshape(T, H, d), eps)
    k = rms(linear(x, W[pre + "k"]).reshape(T, G, d), eps)
    v = linear(x, W[pre + "v"]).reshape(T, G, dv)
    heads = attend_with_one_more(q, k, v, m["scale"], chunk_mask(T, (m.get("mask") or {}).get("size", 0)))
    return linear(heads.reshape(T, H * dv), W[pre + "o"])


# --------------------------------------------------------------------------- recurrences
def retention_scan(q: Tensor, k: Tensor, v: Tensor, decay: List[float]) -> Tensor:
    """q, k [T, H, d], v [T, H, dv]: S <- decay_h S + k v^T; o = S^T q, from a zero state."""
    T, H, d = q.shape
    o = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=q.dtype)
        for t in range(T):
            S = decay[h] * S + torch.outer(k[t, h], v[t, h])
            o[t, h] = q[t, h] @ S
    return o


def retention(x: Tensor, W: Dict[str, Tensor], pre: str, m: dict, eps: float, positions: Tensor) -> Tensor:
    T = x.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    freq = frequencies(rot["dims"], rot["base"])
    q = rotate(linear(x, W[pre + "q"]).reshape(T, H, d), positions, freq, True)
    k = rotate(linear(x, W[pre + "k"]).reshape(T, H, d), positions, freq, True) * d ** -0.5
    v = linear(x, W[pre + "v"]).reshape(T, H, dv)
    o = rms(retention_scan(q, k, v, m["decay"]), eps).reshape(T, H * dv)
    return linear(o * silu(linear(x, W[pre + "g"])), W[pre + "o"])


def parallel(x: Tensor, W: Dict[str, Tensor], pre: str, m: dict, eps: float, positions: Tensor) -> Tensor:
    left = chunked_attention(x, W, pre + "left.", m["left"], eps)
    right = retention(x, W, pre + "right.", m["right"], eps, positions)
    return 0.5 * (rms(left, eps) * W[pre + "left.out"] + rms(right, eps) * W[pre + "right.out"])


def shifted_mix(x: Tensor, mu: Tensor) -> Tensor:
    """x_t + (x_(t-1) - x_t) mu, zeros before the first token."""
    before = torch.cat([torch.zeros_like(x[:1]), x[:-1]], dim=0)
    return x + (before - x) * mu


def wkv_scan(r: Tensor, k: Tensor, v: Tensor, w: Tensor, u: Tensor) -> Tensor:
    """r, k, v, w [T, H, d], u [H, d]: o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T, from a zero state."""
    T, H, d = r.shape
    o = torch.zeros(T, H, v.shape[2], dtype=r.dtype)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=r.dtype)
        for t in range(T):
            kv = torch.outer(k[t, h], v[t, h])
            o[t, h] = r[t, h] @ (S + u[h][:, None] * kv)
            S = w[t, h][:, None] * S + kv
    return o


def wkv(x: Tensor, W: Dict[str, Tensor], pre: str, m: dict, eps: float) -> Tensor:
    T = x.shape[0]
    H, d = m["heads"], m["dim"]
    r, k, v = (linear(shifted_mix(x, W[pre + "mu." + s]), W[pre + s]).reshape(T, H, d) for s in ("r", "k", "v"))
    gate = silu(linear(shifted_mix(x, W[pre + "mu.g"]), W[pre + "g"]))
    low = torch.tanh(linear(shifted_mix(x, W[pre + "mu.w"]), W[pre + "w1"]))
    w = torch.exp(-torch.exp(linear(low, W[pre + "w2"]) + W[pre + "w0"])).reshape(T, H, d)
    o = rms(wkv_scan(r, k, v, w, W[pre + "u"]), eps).reshape(T, H * d)
    return linear(o * W[pre + "norm"] * gate, W[pre + "o"])


# --------------------------------------------------------------------------- the model
def feed_forward(x: Tensor, W: Dict[str, Tensor], pre: str) -> Tensor:
    return linear(gelu_erf(linear(x, W[pre + "up"])), W[pre + "down"])


def forward(config: dict, W: Dict[str, Tensor], tokens: List[int], dtype=torch.float64, layers_out: Optional[list] = None) -> Tensor:
    """Logits [T, vocab] of one sequence from position 0.  ``layers_out``: a list that receives the stream after every
    layer."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in W.items()}
    eps, mult = config["norm"]["eps"], config["residual_mult"]
    positions = torch.arange(len(tokens))
    x = embed(tokens, W, (config.get("embedding") or {}).get("bigram"))
    shared: dict = {}
    for i, layer in enumerate(config["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        h = norm(x, W[pre + "norm1"], eps)
        if layer["type"] == "attention":
            y = attention(h, W, pre + "mix.", m, eps, positions, shared)
        elif layer["type"] == "parallel":
            y = parallel(h, W, pre + "mix.", m, eps, positions)
        elif layer["type"] == "wkv":
            y = wkv(h, W, pre + "mix.", m, eps)
        else:
            raise ValueError(f"unknown layer type {layer['type']}")
        x = x + mult * norm(y, W[pre + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(norm(x, W[pre + "norm2"], eps), W, pre + "mlp.")
            x = x + mult * norm(y, W[pre + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(norm(x, W["final.norm"], eps), W["head"])
