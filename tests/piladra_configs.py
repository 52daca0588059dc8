"""Tiny Piladra configurations of the test-suite and model folders with random weights for them.

They differ in every size and option: widths that are and are not multiples of 8; norms over one, several and many
groups; input convolutions of one to six taps; loops that cover the whole model, its middle, one layer, and none, run
once, twice and three times; attention with one key/value head, several and as many as query heads, key sizes above and
below the value sizes, rotation of the whole head, of a part and none, with and without scaled frequencies (whose
blended band holds several, one and no frequency), windows shorter and longer than a page and none; latent layers
whose cache row is padded to 32, 64, 128 and 144 entries; scans with state sizes of 1 to 40, step-size ranks that are
and are not multiples of 8, convolutions of one to five taps; dense, routed and no feed-forward, with and without a
shared expert, one expert a token, several and all; residual multipliers below, at and above one; with and without a
softcap.
"""
from __future__ import annotations

import copy
import json
import math
import os
import random
from typing import Dict, List, Tuple

import torch


def attention(heads, kv_heads, dim, vdim, scale, rot=None, scaling=None, window=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if window is not None:
        m["mask"] = {"size": window}
    return m


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
            "rot": {"dims": rot_dim, "base": base}}


def scan(inner, state, dt_rank, conv):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def layer(mixer, mlp):
    kind = "latent_attention" if "kv_rank" in mixer else "mamba1" if "inner" in mixer else "attention"
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


PL_A = {
    "architecture": "Piladra", "vocab": 211, "width": 72, "norm": {"eps": 1e-5, "groups": 3}, "canon": {"taps": 4},
    "residual_mult": 0.7, "logit_softcap": 20.0, "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [
        layer(scan(80, 12, 5, 3), moe(6, 2, 40, shared=24)),
        layer(attention(4, 2, 24, 16, 0.2, rot=(16, 1000.0), scaling=(8.0, 1.0, 4.0, 64), window=24), dense(88)),
        layer(latent(3, 16, 12, 24, 20, 0.25, 5000.0), moe(5, 3, 16)),
        layer(attention(6, 6, 8, 20, 0.35, rot=(8, 50.0), window=40), None),
    ],
}

PL_B = {
    "architecture": "Piladra", "vocab": 130, "width": 100, "norm": {"eps": 1e-6, "groups": 5}, "canon": {"taps": 2},
    "residual_mult": 1.0, "logit_softcap": 8.0, "loop": {"start": 0, "stop": 3, "times": 2},
    "layers": [
        layer(latent(2, 32, 20, 16, 100, 0.15, 300.0), moe(8, 1, 24, shared=40)),
        layer(attention(4, 1, 40, 40, 0.16, rot=(40, 1e5), scaling=(4.0, 1.0, 3.0, 500), window=17), dense(52)),
        layer(scan(64, 16, 8, 4), moe(9, 9, 20)),
    ],
}

PL_C = {
    "architecture": "Piladra", "vocab": 97, "width": 44, "norm": {"eps": 1e-4, "groups": 1}, "canon": {"taps": 6},
    "residual_mult": 0.25,
    "layers": [
        layer(attention(3, 3, 16, 8, 0.3, window=5), moe(4, 3, 12)),
        layer(scan(50, 40, 11, 1), dense(36)),
        layer(latent(1, 8, 4, 12, 140, 0.4, 10.0), None),
        layer(scan(24, 1, 16, 5), moe(12, 4, 8, shared=16)),
        layer(attention(6, 2, 8, 8, 0.35, rot=(4, 20.0)), dense(20)),
    ],
}

# Sizes at which the tensor-core forms of the kernels are the ones that run: cache rows and heads of 64 and 128
# entries, prompts long enough for the tcgen05 attention and for scans in chunks, expert rows of whole 128-byte pieces.
PL_M = {
    "architecture": "Piladra", "vocab": 1000, "width": 384, "norm": {"eps": 1e-6, "groups": 4}, "canon": {"taps": 3},
    "residual_mult": 0.4, "logit_softcap": 25.0, "loop": {"start": 1, "stop": 4, "times": 2},
    "layers": [
        layer(attention(8, 2, 64, 64, 0.125, rot=(64, 1e4), scaling=(4.0, 1.0, 4.0, 256), window=200), dense(512)),
        layer(latent(8, 48, 16, 32, 112, 0.125, 100000.0), moe(8, 2, 128, shared=192)),
        layer(scan(512, 16, 24, 4), moe(16, 3, 64)),
        layer(attention(4, 1, 128, 128, 0.09, rot=(64, 50000.0), window=90), dense(256)),
    ],
}

CONFIGS = {"A": PL_A, "B": PL_B, "C": PL_C, "M": PL_M}


def config(which: str) -> dict:
    return copy.deepcopy(CONFIGS[which])


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """name -> float32 tensor of bfloat16-representable values, written from the names and shapes the architecture's
    tensors have (no package code): matrices N(0, gain / in), so that every branch of a layer carries weight in the
    logits; norm weights around one, sinks and convolution taps of order one, decays from slow to fast."""
    g = torch.Generator().manual_seed(seed)
    D, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    W: Dict[str, torch.Tensor] = {}

    def mat(name, out, inp, gain=1.0):
        W[name] = torch.randn(out, inp, generator=g) * (gain / math.sqrt(inp))

    def vec(name, shape, std=1.0, mean=0.0):
        W[name] = torch.randn(shape, generator=g) * std + mean

    def ffn(p, ff):
        mat(p + "gate", ff, D, 1.2)
        mat(p + "up", ff, D, 1.2)
        mat(p + "down", D, ff)

    vec("embed", (V, D), 1.0)
    mat("head", V, D, 1.5)
    vec("final.norm", (D,), 0.2, 1.0)
    if cfg.get("loop") is not None:
        vec("loop.step", (cfg["loop"]["times"], D), 0.7)
    for i, lay in enumerate(cfg["layers"]):
        p = f"l{i}."
        m = lay["mixer"]
        vec(p + "norm1", (D,), 0.2, 1.0)
        vec(p + "canon1", (D, taps), 0.4)
        if lay["type"] == "latent_attention":
            H, d, rd, dv, rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            mat(p + "mix.q", H * (d + rd), D, 1.5)
            mat(p + "mix.dkv", rk + rd, D, 1.5)
            vec(p + "mix.dkv.norm", (rk,), 0.2, 1.0)
            mat(p + "mix.uk", H * d, rk, 1.5)
            mat(p + "mix.uv", H * dv, rk, 1.2)
            mat(p + "mix.g", H * dv, D, 2.0)
            mat(p + "mix.o", D, H * dv)
        elif lay["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            mat(p + "mix.q", H * d, D, 1.5)
            mat(p + "mix.k", G * d, D, 1.5)
            mat(p + "mix.v", G * dv, D, 1.5)
            vec(p + "mix.sink", (H,), 1.0, 0.5)
            mat(p + "mix.o", D, H * dv)
        else:
            I, N, R = m["inner"], m["state"], m["dt_rank"]
            mat(p + "mix.in", 2 * I, D, 1.2)
            vec(p + "mix.conv", (I, m["conv"]), 0.5)
            vec(p + "mix.conv.b", (I,), 0.3)
            mat(p + "mix.x", R + 2 * N, I, 1.0)
            mat(p + "mix.dt", I, R, 1.0)
            vec(p + "mix.dt.b", (I,), 0.8, -2.0)
            W[p + "mix.A_log"] = torch.rand(I, N, generator=g) * 3.5 - 2.0
            vec(p + "mix.D", (I,), 0.3, 0.7)
            mat(p + "mix.o", D, I, 1.0)
        mlp = lay.get("mlp")
        if mlp is None:
            continue
        vec(p + "norm2", (D,), 0.2, 1.0)
        vec(p + "canon2", (D, taps), 0.4)
        if mlp["kind"] == "dense":
            ffn(p + "mlp.", mlp["ff"])
            continue
        E = mlp["router"]["experts"]
        mat(p + "mlp.router", E, D, 1.5)
        for e in range(E):
            ffn(p + f"mlp.e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared") is not None:
            ffn(p + "mlp.shared.", mlp["shared"]["ff"])
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in W.items()}


def make_model_dir(which, out_dir: str, seed: int = 0, patch=None, edit=None) -> Tuple[str, dict, Dict[str, torch.Tensor]]:
    """(folder, config dict, float32 weights by name).  ``patch(cfg)`` changes the configuration before the weights are
    made, ``edit(weights)`` the weights before they are stored."""
    from poor_mans_mamba_b200.weights import save_file
    cfg = config(which) if isinstance(which, str) else copy.deepcopy(which)
    if patch:
        patch(cfg)
    weights = make_weights(cfg, seed)
    if edit:
        edit(weights)
        weights = {k: v.to(torch.bfloat16).to(torch.float32) for k, v in weights.items()}
    os.makedirs(out_dir, exist_ok=True)
    with open(os.path.join(out_dir, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    save_file({k: v.to(torch.bfloat16) for k, v in weights.items()}, os.path.join(out_dir, "model.safetensors"))
    return out_dir, cfg, weights


def decisive_routers(weights: Dict[str, torch.Tensor]) -> None:
    """Routers whose choice no rounding can turn.  The first channel of the stream is made a positive constant of the
    token (the same large entry in every row of the embedding table; nothing writes to it: the first row of every output
    matrix and the first entry of every pass's vector are zero), and the input convolutions leave it alone, so the
    first entry of what a router reads is positive and well away from zero.  The first column of every router is an
    evenly spaced permutation around zero and the rest of it small, so that the experts' logits lie about evenly spaced
    in an order that is the same for every token of the layer, with scores that still depend on the token.  bfloat16
    runs are compared with the plain implementation under such routers: with freely routed tokens a few per cent of
    them choose between two experts whose scores differ by less than bfloat16 rounding moves them, and either choice
    is right."""
    weights["embed"][:, 0] = 6.0
    for name in sorted(weights):
        w = weights[name]
        if name.endswith((".mix.o", ".down")):
            w[0, :] = 0.0
        elif name == "loop.step":
            w[:, 0] = 0.0
        elif name.endswith(("canon1", "canon2")):
            w[0, :] = 0.0
        elif name.endswith("norm2"):
            w[0] = 1.0
        elif name.endswith("mlp.router"):
            E = w.shape[0]
            order = torch.randperm(E, generator=torch.Generator().manual_seed(len(name) + E)).to(torch.float32)
            w[:, 1:] *= 0.02
            w[:, 0] = (order - (E - 1) / 2) * (6.0 / E)


def sequences(cfg: dict, lengths, seed: int = 0) -> List[List[int]]:
    rng = random.Random(seed)
    return [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in lengths]
