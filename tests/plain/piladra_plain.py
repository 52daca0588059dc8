"""Plain, slow Piladra forward pass: whole sequences, no cache, one function per mechanism.

The oracle of the Piladra tests.  It shares no code with the package: the configuration is a plain
dict, the weights a ``name -> tensor`` dict, and every formula runs directly on the CPU in one
floating-point type (float64 by default).  Notation: T tokens, D model width, linear weights stored
[out, in].  Keys and values of the latent mixer are made for every token and head from its latent
(nothing is moved to the query side), masks are dense T x T tables, convolutions are loops over taps,
the selective scan and the router loops over tokens, and an expert really receives its weighted input.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensor = torch.Tensor


# --------------------------------------------------------------------------- small functions
def linear(x: Tensor, w: Tensor) -> Tensor:
    return x @ w.t()


def silu(z: Tensor) -> Tensor:
    return z * torch.sigmoid(z)


def softplus(z: Tensor) -> Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def rms(x: Tensor, eps: float) -> Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def grouped_norm(x: Tensor, w: Tensor, eps: float, groups: int) -> Tensor:
    """The last axis in ``groups`` equal neighbouring parts, each over its own root mean square; then times w."""
    T, D = x.shape
    return rms(x.reshape(T, groups, D // groups), eps).reshape(T, D) * w


def causal_conv(u: Tensor, w: Tensor) -> Tensor:
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, _ = u.shape
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        shift = taps - 1 - j
        if shift < T:
            y[shift:] += u[:T - shift] * w[:, j]
    return y


def input_conv(h: Tensor, w: Tensor) -> Tensor:
    return h + causal_conv(h, w)


# --------------------------------------------------------------------------- positions
def frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> Tensor:
    """f_i = base^(-2i/dims); with ``scaling`` long wavelengths are stretched by ``factor``, short ones
    kept, and those between original/high and original/low blended linearly in original/wavelength."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            wave = 2.0 * math.pi / f
            n = scaling["original"] / wave
            if n < scaling["low"]:
                f = f / scaling["factor"]
            elif n <= scaling["high"]:
                s = (n - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_halves(x: Tensor, positions: Tensor, freq: Tensor) -> Tensor:
    """x [T, ..., d]: among the first dims = 2 len(freq) entries, entry i and entry i + dims/2 turn together."""
    half = freq.shape[0]
    if half == 0:
        return x.clone()
    ang = positions.to(torch.float64)[:, None] * freq[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [half]
    c, s = torch.cos(ang).to(x.dtype).reshape(shape), torch.sin(ang).to(x.dtype).reshape(shape)
    out = x.clone()
    u, v = x[..., :half], x[..., half:2 * half]
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


# --------------------------------------------------------------------------- softmax attention
def window_mask(T: int, size: int) -> Tensor:
    """[T, T] bool: i sees j when 0 <= i - j < size (size 0: every j <= i)."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size > 0 else torch.ones(T, T, dtype=torch.bool))


def masked_softmax_attention(q: Tensor, k: Tensor, v: Tensor, scale: float, mask: Tensor, sink: Optional[Tensor]) -> Tensor:
    """q, k [T, H, d], v [T, H, dv]; ``sink`` [H]: the denominator of head h also holds exp(sink[h])."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        s = ((q[:, h] @ k[:, h].t()) * scale).masked_fill(~mask, -math.inf)
        m = s.max(dim=-1, keepdim=True).values
        if sink is not None:
            m = torch.maximum(m, sink[h].expand_as(m))
        p = torch.exp(s - m)
        den = p.sum(dim=-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - m)
        out[:, h] = (p / den) @ v[:, h]
    return out


# --------------------------------------------------------------------------- mixers
def attention(x: Tensor, W: Dict[str, Tensor], pre: str, m: dict, eps: float, positions: Tensor) -> Tensor:
    """Grouped queries, scaled rotation, unit-rms values, a sliding window and a sink per head."""
    T = x.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    freq = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    q = rotate_halves(linear(x, W[pre + "q"]).reshape(T, H, d), positions, freq)
    k = rotate_halves(linear(x, W[pre + "k"]).reshape(T, G, d), positions, freq)
    v = rms(linear(x, W[pre + "v"]).reshape(T, G, dv), eps)
    rep = H // G
    mask = window_mask(T, (m.get("mask") or {}).get("size", 0))
    heads = masked_softmax_attention(q, k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1), m["scale"], mask,
                                     W[pre + "sink"])
    return linear(heads.reshape(T, H * dv), W[pre + "o"])


def latent_attention(x: Tensor, W: Dict[str, Tensor], pre: str, m: dict, eps: float, positions: Tensor) -> Tensor:
    """Keys and values from a normed latent, one rotated key part for all heads, every earlier token visible,
    and a sigmoid gate per channel of the concatenated heads."""
    T = x.shape[0]
    H, d, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    freq = frequencies(m["rot"]["dims"], m["rot"]["base"])
    q = linear(x, W[pre + "q"]).reshape(T, H, d + dr)
    low = linear(x, W[pre + "dkv"])
    c = rms(low[:, :R], eps) * W[pre + "dkv.norm"]
    r = rotate_halves(low[:, R:], positions, freq)
    q_full = torch.cat([q[..., :d], rotate_halves(q[..., d:], positions, freq)], dim=-1)
    k_full = torch.cat([linear(c, W[pre + "uk"]).reshape(T, H, d), r[:, None, :].expand(T, H, dr)], dim=-1)
    v = linear(c, W[pre + "uv"]).reshape(T, H, dv)
    heads = masked_softmax_attention(q_full, k_full, v, m["scale"], window_mask(T, 0), None)
    return linear(heads.reshape(T, H * dv) * torch.sigmoid(linear(x, W[pre + "g"])), W[pre + "o"])


def selective_scan(x: Tensor, dt: Tensor, A: Tensor, B: Tensor, C: Tensor, D: Tensor) -> Tensor:
    """x, dt [T, I], A [I, N], B, C [T, N], D [I]: S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;
    y_c = sum_n S[c, n] C_n + D_c x_c, token by token from a zero state."""
    S = torch.zeros_like(A)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def mamba1(h: Tensor, W: Dict[str, Tensor], pre: str, m: dict) -> Tensor:
    I, N, R = m["inner"], m["state"], m["dt_rank"]
    xz = linear(h, W[pre + "in"])
    x, z = xz[:, :I], xz[:, I:]
    x = silu(causal_conv(x, W[pre + "conv"]) + W[pre + "conv.b"])
    low = linear(x, W[pre + "x"])
    dt = softplus(linear(low[:, :R], W[pre + "dt"]) + W[pre + "dt.b"])
    y = selective_scan(x, dt, -torch.exp(W[pre + "A_log"]), low[:, R:R + N], low[:, R + N:], W[pre + "D"])
    return linear(y * silu(z), W[pre + "o"])


# --------------------------------------------------------------------------- feed-forward
def gated_ffn(x: Tensor, W: Dict[str, Tensor], pre: str) -> Tensor:
    return linear(silu(linear(x, W[pre + "gate"])) * linear(x, W[pre + "up"]), W[pre + "down"])


def route(z: Tensor, top: int):
    """z [E] -> (chosen experts, their weights): the ``top`` largest sigmoids, as they are."""
    s = torch.sigmoid(z)
    chosen = sorted(range(z.shape[0]), key=lambda e: (-float(s[e]), e))[:top]
    return chosen, [s[e] for e in chosen]


def routed_ffn(x: Tensor, W: Dict[str, Tensor], pre: str, mlp: dict) -> Tensor:
    z = linear(x, W[pre + "router"])
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e, w in zip(*route(z[t], mlp["router"]["top"])):
            out[t] += gated_ffn(w * x[t:t + 1], W, f"{pre}e{e}.")[0]
    if mlp.get("shared") is not None:
        out = out + gated_ffn(x, W, pre + "shared.")
    return out


# --------------------------------------------------------------------------- the model
def layer_runs(config: dict):
    """[(layer, pass number if this run begins a pass else None)] in the order they run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if loop is None:
        return [(i, None) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, None) for i in range(a)]
    for t in range(times):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(config: dict, W: Dict[str, Tensor], tokens: List[int], dtype=torch.float64, layers_out: Optional[list] = None) -> Tensor:
    """Logits [T, vocab] of one sequence from position 0.  ``layers_out``: a list that receives the stream
    after every layer run."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in W.items()}
    eps, groups, mult = config["norm"]["eps"], config["norm"]["groups"], config["residual_mult"]
    T = len(tokens)
    positions = torch.arange(T)
    x = W["embed"][torch.tensor(tokens)]
    for i, begins in layer_runs(config):
        pre, layer = f"l{i}.", config["layers"][i]
        m = layer["mixer"]
        if begins is not None:
            x = x + W["loop.step"][begins]
        h = input_conv(grouped_norm(x, W[pre + "norm1"], eps, groups), W[pre + "canon1"])
        if layer["type"] == "attention":
            y = attention(h, W, pre + "mix.", m, eps, positions)
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, W, pre + "mix.", m, eps, positions)
        elif layer["type"] == "mamba1":
            y = mamba1(h, W, pre + "mix.", m)
        else:
            raise ValueError(f"unknown layer type {layer['type']}")
        x = x + mult * y
        mlp = layer.get("mlp")
        if mlp is not None:
            h = input_conv(grouped_norm(x, W[pre + "norm2"], eps, groups), W[pre + "canon2"])
            y = gated_ffn(h, W, pre + "mlp.") if mlp["kind"] == "dense" else routed_ffn(h, W, pre + "mlp.", mlp)
            x = x + mult * y
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = linear(grouped_norm(x, W["final.norm"], eps, groups), W["head"])
    cap = config.get("logit_softcap")
    return logits if not cap else cap * torch.tanh(logits / cap)
