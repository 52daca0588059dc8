"""Tiny Nikodra configurations of the test-suite and model folders with random weights for them.

They differ in every size and option: widths that are and are not multiples of 8; with and without a bigram table, whose
multipliers are small, zero and large; attention with one key/value head, several and as many as query heads, key sizes
above and below the value sizes, rotation of the whole head, of a part and none, with and without scaled frequencies
(whose blended band holds several, one and no pair), values mixed in several layers, in one only and in none, first and
late in the model; chunks shorter than, equal to and longer than a page, of one token, and none; retention with rotation
of the whole head, a part and none, decays from fast to none at all; time mixing with decays from instant to almost
none, ranks that are and are not multiples of 8; layers without a feed-forward; residual multipliers below, at and above
one.
"""
from __future__ import annotations

import copy
import json
import math
import os
import random
from typing import Dict, List, Tuple

import torch


def attention(heads, kv_heads, dim, vdim, scale, rot=None, yarn=None, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if yarn is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return m


def parallel(left, right):
    """left: (heads, kv_heads, dim, vdim, scale, chunk or None); right: (dim, vdim, decays, rotation or None)."""
    l = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left))
    if left[5] is not None:
        l["mask"] = {"size": left[5]}
    r = {"heads": len(right[2]), "dim": right[0], "vdim": right[1], "decay": list(right[2])}
    if right[3] is not None:
        r["rot"] = {"dims": right[3][0], "base": right[3][1]}
    return {"left": l, "right": r}


def wkv(heads, dim, rank):
    return {"heads": heads, "dim": dim, "decay_rank": rank}


def layer(mixer, ff):
    kind = "parallel" if "left" in mixer else "wkv" if "decay_rank" in mixer else "attention"
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


NK_A = {
    "architecture": "Nikodra", "vocab": 211, "width": 72, "norm": {"eps": 1e-5}, "residual_mult": 0.6,
    "embedding": {"bigram": {"buckets": 101, "mul_prev": 31, "mul_cur": 3}},
    "layers": [
        layer(attention(6, 2, 24, 16, 0.25, rot=(16, 1000.0), yarn=(4.0, 64, 8.0, 1.0)), 88),
        layer(parallel((4, 2, 16, 24, 0.3, 24), (12, 20, (0.5, 0.9, 0.99), (8, 50.0))), 40),
        layer(wkv(3, 16, 5), 100),
        layer(attention(2, 2, 40, 16, 0.2, rot=(40, 5000.0)), None),
        layer(attention(4, 1, 8, 8, 0.4, rot=(4, 20.0), v_mix=False), 24),
    ],
}

NK_B = {
    "architecture": "Nikodra", "vocab": 130, "width": 100, "norm": {"eps": 1e-6}, "residual_mult": 1.0,
    "embedding": {"bigram": {"buckets": 17, "mul_prev": 100003, "mul_cur": 0}},
    "layers": [
        layer(wkv(2, 40, 24), None),
        layer(attention(3, 3, 16, 32, 0.3, v_mix=False), 52),
        layer(parallel((6, 1, 48, 16, 0.2, 64), (32, 16, (0.97, 0.999), (32, 1e5))), 60),
        layer(attention(4, 1, 32, 40, 0.2, rot=(32, 1e5), yarn=(16.0, 300, 32.0, 1.0)), 64),
        layer(wkv(5, 12, 8), 36),
        layer(attention(2, 1, 20, 40, 0.3, rot=(8, 400.0), yarn=(2.0, 40, 1.0, 1.0)), 44),
    ],
}

NK_C = {
    "architecture": "Nikodra", "vocab": 97, "width": 44, "norm": {"eps": 1e-4}, "residual_mult": 1.2,
    "layers": [
        layer(parallel((3, 3, 8, 12, 0.4, 5), (16, 8, (1.0, 0.3, 0.8, 0.95), None)), 36),
        layer(wkv(1, 64, 3), 20),
        layer(parallel((2, 2, 12, 8, 0.5, 40), (8, 24, (0.9,), (6, 10.0))), None),
        layer(attention(6, 2, 16, 8, 0.35, rot=(8, 20.0)), 48),
        layer(parallel((4, 2, 8, 8, 0.4, None), (4, 4, (0.7, 0.98), (4, 100.0))), 28),
        layer(parallel((2, 1, 16, 16, 0.3, 1), (20, 12, (0.99, 0.6), (2, 3.0))), 16),
    ],
}

# Sizes at which the tensor-core forms of the kernels are the ones that run: heads of 64 and 128 entries, prompts long
# enough for the tcgen05 attention and for recurrences in chunks.
NK_M = {
    "architecture": "Nikodra", "vocab": 1000, "width": 384, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
    "embedding": {"bigram": {"buckets": 4099, "mul_prev": 911, "mul_cur": 13}},
    "layers": [
        layer(attention(8, 2, 64, 64, 0.125, rot=(64, 1e4), yarn=(8.0, 256, 32.0, 1.0)), 512),
        layer(parallel((8, 2, 64, 48, 0.2, 200), (64, 128, (0.9, 0.97, 0.99, 0.999), (64, 1e5))), 768),
        layer(wkv(6, 64, 32), 640),
        layer(attention(4, 2, 128, 64, 0.09, rot=(64, 50000.0)), 256),
        layer(parallel((4, 1, 128, 128, 0.1, 64), (128, 64, (0.95, 0.998), (128, 1e6))), 512),
    ],
}

CONFIGS = {"A": NK_A, "B": NK_B, "C": NK_C, "M": NK_M}


def config(which: str) -> dict:
    return copy.deepcopy(CONFIGS[which])


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """name -> float32 tensor of bfloat16-representable values, written from the names and shapes the architecture's
    tensors have (no package code): matrices N(0, gain / in), so that every branch of a layer carries weight in the
    logits; norm weights and biases that are felt, mixes and decays over their whole range."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    W: Dict[str, torch.Tensor] = {}

    def mat(name, out, inp, gain=1.0):
        W[name] = torch.randn(out, inp, generator=g) * (gain / math.sqrt(inp))

    def vec(name, shape, std=1.0, mean=0.0):
        W[name] = torch.randn(shape, generator=g) * std + mean

    def uniform(name, shape, lo, hi):
        W[name] = lo + (hi - lo) * torch.rand(shape, generator=g)

    vec("embed", (V, D), 1.0)
    bigram = (cfg.get("embedding") or {}).get("bigram")
    if bigram is not None:
        vec("bigram", (bigram["buckets"] + 1, D), 0.8)
    mat("head", V, D, 1.5)
    vec("final.norm", (D,), 0.2)
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        x = p + "mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if lay["mlp"] else ()):
            vec(p + n, (D,), 0.3)
        if lay["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                mat(x + n, rows, D, 1.3)
                vec(x + n + ".b", (rows,), 0.4)
            uniform(x + "q.norm", (d,), 0.4, 2.2)
            uniform(x + "k.norm", (d,), 0.4, 2.2)
            if m.get("v_mix"):
                uniform(x + "vmix", (), 0.3, 0.7)
            mat(x + "o", D, H * dv)
            vec(x + "o.b", (D,), 0.4)
        elif lay["type"] == "parallel":
            l, r = m["left"], m["right"]
            mat(x + "left.q", l["heads"] * l["dim"], D)
            mat(x + "left.k", l["kv_heads"] * l["dim"], D)
            mat(x + "left.v", l["kv_heads"] * l["vdim"], D, 1.3)
            mat(x + "left.o", D, l["heads"] * l["vdim"])
            vec(x + "left.out", (D,), 0.3, 1.0)
            for n, rows in (("q", r["dim"]), ("k", r["dim"]), ("v", r["vdim"]), ("g", r["vdim"])):
                mat(x + "right." + n, r["heads"] * rows, D, 1.2)
            mat(x + "right.o", D, r["heads"] * r["vdim"])
            vec(x + "right.out", (D,), 0.3, 1.0)
        else:
            H, d, rank = m["heads"], m["dim"], m["decay_rank"]
            for n in ("r", "k", "v", "g", "w"):
                uniform(x + "mu." + n, (D,), -0.2, 1.2)
            for n in ("r", "k", "v", "g"):
                mat(x + n, H * d, D, 1.2)
            mat(x + "w1", rank, D, 1.2)
            mat(x + "w2", H * d, rank, 1.0)
            uniform(x + "w0", (H * d,), -6.0, 1.5)
            vec(x + "u", (H, d), 0.8, 0.5)
            vec(x + "norm", (H * d,), 0.3, 1.0)
            mat(x + "o", D, H * d)
        if lay["mlp"]:
            mat(p + "mlp.up", lay["mlp"]["ff"], D, 1.5)
            mat(p + "mlp.down", D, lay["mlp"]["ff"])
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in W.items()}


def make_model_dir(which, out_dir: str, seed: int = 0, patch=None, edit=None) -> Tuple[str, dict, Dict[str, torch.Tensor]]:
    """(folder, config dict, float32 weights by name).  ``patch(cfg)`` changes the configuration before the weights are
    made, ``edit(weights)`` the weights before they are stored.  The folder's config.json does not say the ranks of the
    low-rank decays: the tensors' shapes do."""
    from poor_mans_mamba_b200.weights import save_file
    cfg = config(which) if isinstance(which, str) else copy.deepcopy(which)
    if patch:
        patch(cfg)
    weights = make_weights(cfg, seed)
    if edit:
        edit(weights)
        weights = {k: v.to(torch.bfloat16).to(torch.float32) for k, v in weights.items()}
    os.makedirs(out_dir, exist_ok=True)
    stored = copy.deepcopy(cfg)
    for lay in stored["layers"]:
        lay["mixer"].pop("decay_rank", None)
    with open(os.path.join(out_dir, "config.json"), "w") as fh:
        json.dump(stored, fh)
    save_file({k: v.to(torch.bfloat16) for k, v in weights.items()}, os.path.join(out_dir, "model.safetensors"))
    return out_dir, cfg, weights


def sequences(cfg: dict, lengths, seed: int = 0) -> List[List[int]]:
    rng = random.Random(seed)
    return [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in lengths]
