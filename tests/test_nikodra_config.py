"""Nikodra's configuration reader, its description as parts, its tensor names, what the cache manager keeps for it, and
the plain implementation's own pieces on cases done by hand (no GPU)."""
import json
import math
import os

import pytest
import torch

import nikodra_configs as C
from plain import nikodra_plain as P

import poor_mans_mamba_b200.architectures  # noqa: F401  (registration)
from poor_mans_mamba_b200.cache import CacheManager
from poor_mans_mamba_b200.config import ConfigError, resolve_architecture
from poor_mans_mamba_b200.config.nikodra import NikodraConfig
from poor_mans_mamba_b200.config.registry import open_model_dir
from poor_mans_mamba_b200.engine.model import Model
from poor_mans_mamba_b200.engine.scheduler import SamplingParams, Scheduler
from poor_mans_mamba_b200.parts.base import EMBEDDING_CACHE
from poor_mans_mamba_b200.parts.rope import yarn_frequencies
from poor_mans_mamba_b200.weights import write_random_model
from poor_mans_mamba_b200.weights.loader import check_tensors
from poor_mans_mamba_b200.weights.safetensors_io import ModelFiles

F64 = torch.float64


@pytest.mark.parametrize("which", ["A", "B", "C", "M"])
def test_every_size_and_constant_is_read(which):
    data = C.config(which)
    cfg = NikodraConfig.from_dict(data)
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.residual_mult) == (
        data["vocab"], data["width"], data["norm"]["eps"], data["residual_mult"])
    b = (data.get("embedding") or {}).get("bigram")
    if b is None:
        assert cfg.bigram is None
    else:
        assert (cfg.bigram.buckets, cfg.bigram.mul_prev, cfg.bigram.mul_cur) == (b["buckets"], b["mul_prev"], b["mul_cur"])
    for l, raw in zip(cfg.layers, data["layers"]):
        m = raw["mixer"]
        assert l.type == raw["type"] and l.ff == (None if raw["mlp"] is None else raw["mlp"]["ff"])
        assert [x is not None for x in (l.attention, l.left, l.right, l.wkv)] == [
            raw["type"] == t for t in ("attention", "parallel", "parallel", "wkv")]
        if l.attention is not None:
            x, rot = l.attention, m.get("rot") or {"dims": 0, "base": 1.0}
            assert (x.heads, x.kv_heads, x.dim, x.vdim, x.scale, x.v_mix) == tuple(
                m[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale", "v_mix"))
            assert (x.rot_dims, x.rot_base) == (rot["dims"], rot["base"])
            s = rot.get("scaling")
            assert x.rot_scaling == (None if s is None else tuple(s[k] for k in ("factor", "original", "fast", "slow")))
        elif l.wkv is not None:
            assert (l.wkv.heads, l.wkv.dim, l.wkv.decay_rank) == (m["heads"], m["dim"], m["decay_rank"])
        else:
            x, y = l.left, l.right
            assert (x.heads, x.kv_heads, x.dim, x.vdim, x.scale) == tuple(
                m["left"][k] for k in ("heads", "kv_heads", "dim", "vdim", "scale"))
            assert x.chunk == m["left"].get("mask", {}).get("size", 0)
            rot = m["right"].get("rot") or {"dims": 0, "base": 1.0}
            assert (y.heads, y.dim, y.vdim, list(y.decay), y.rot_dims, y.rot_base) == (
                *(m["right"][k] for k in ("heads", "dim", "vdim", "decay")), rot["dims"], rot["base"])


def test_the_architecture_is_chosen_by_its_name():
    assert resolve_architecture(C.config("A")).name == "Nikodra"


@pytest.mark.parametrize("path,value,needle", [
    (("width",), 0, "width"), (("vocab",), -3, "vocab"),
    (("embedding", "bigram", "buckets"), 0, "embedding.bigram.buckets"),
    (("embedding", "bigram", "mul_prev"), -1, "embedding.bigram.mul_prev"),
    (("layers", 0, "type"), "mamba", "layers[0].type"),
    (("layers", 0, "mixer", "kv_heads"), 4, "layers[0].mixer.heads"),
    (("layers", 0, "mixer", "rot", "dims"), 7, "layers[0].mixer.rot.dims"),
    (("layers", 0, "mixer", "rot", "dims"), 26, "layers[0].mixer.rot.dims"),
    (("layers", 0, "mixer", "rot", "base"), 1.0, "layers[0].mixer.rot.base"),
    (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0, "layers[0].mixer.rot.scaling"),
    (("layers", 0, "mlp", "kind"), "glu", "layers[0].mlp.kind"),
    (("layers", 0, "mlp", "ff"), 0, "layers[0].mlp.ff"),
    (("layers", 1, "mixer", "left", "mask", "size"), -1, "layers[1].mixer.left.mask.size"),
    (("layers", 1, "mixer", "left", "vdim"), 0, "layers[1].mixer.left.vdim"),
    (("layers", 1, "mixer", "right", "decay"), [0.5, 0.5], "decay"),
    (("layers", 1, "mixer", "right", "rot", "dims"), 14, "layers[1].mixer.right.rot.dims"),
    (("layers", 2, "mixer", "dim"), 0, "layers[2].mixer.dim"),
    (("layers", 3, "mixer", "vdim"), 24, "layers[3].mixer.v_mix"),
])
def test_errors_name_the_key(path, value, needle):
    data = C.config("A")
    node = data
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    with pytest.raises(ConfigError) as exc:
        NikodraConfig.from_dict(data)
    assert needle in str(exc.value)


def test_missing_keys_are_refused_and_optional_ones_default():
    for path in (("residual_mult",), ("norm", "eps"), ("embedding", "bigram", "mul_cur"), ("layers", 0, "mixer", "scale"),
                 ("layers", 0, "mixer", "rot", "scaling", "slow"), ("layers", 1, "mixer", "right", "decay"),
                 ("layers", 2, "mixer", "decay_rank"), ("layers", 1, "mixer", "left", "vdim")):
        data = C.config("A")
        node = data
        for k in path[:-1]:
            node = node[k]
        del node[path[-1]]
        with pytest.raises(ConfigError, match=path[-1]):
            NikodraConfig.from_dict(data)
    data = C.config("A")
    del data["embedding"], data["layers"][1]["mixer"]["left"]["mask"], data["layers"][1]["mixer"]["right"]["rot"]
    del data["layers"][0]["mixer"]["rot"], data["layers"][3]["mixer"]["v_mix"]
    data["layers"][2]["mlp"] = None
    cfg = NikodraConfig.from_dict(data)
    assert cfg.bigram is None and cfg.layers[1].left.chunk == 0 and cfg.layers[1].right.rot_dims == 0
    assert cfg.layers[0].attention.rot_dims == 0 and not cfg.layers[3].attention.v_mix and cfg.layers[2].ff is None


@pytest.mark.parametrize("which", ["A", "B", "C", "M"])
def test_states_of_every_layer_and_of_the_embedding(which):
    data = C.config(which)
    model = Model(resolve_architecture(data).model_spec(NikodraConfig.from_dict(data)))
    states = {k: dict(v) for k, v in model.state_specs().items()}
    assert (EMBEDDING_CACHE in states) == bool(data.get("embedding"))
    if EMBEDDING_CACHE in states:
        assert states[EMBEDDING_CACHE]["bigram.previous"].dtype == "int32"

    def padded(m):
        return m["kv_heads"] * ((max(m["dim"], m["vdim"]) + 15) // 16 * 16)
    for i, raw in enumerate(data["layers"]):
        m, s = raw["mixer"], states[i]
        if raw["type"] == "attention":
            assert set(s) == {"mix.kv"} and (s["mix.kv"].width, s["mix.kv"].window, s["mix.kv"].chunk) == (padded(m), 0, 0)
        elif raw["type"] == "parallel":
            kv, S = s["mix.left.kv"], s["mix.right.S"]
            assert (kv.width, kv.window, kv.chunk) == (padded(m["left"]), 0, m["left"].get("mask", {}).get("size", 0))
            assert S.shape == tuple(m["right"][k] for k in ("heads", "dim", "vdim")) and S.dtype == "float32"
        else:
            assert s["mix.h"].shape == (data["width"],) and s["mix.S"].shape == (m["heads"], m["dim"], m["dim"])
            assert s["mix.h"].dtype == s["mix.S"].dtype == "float32"


def test_a_new_request_starts_from_nothing():
    data = C.config("A")
    model = Model(resolve_architecture(data).model_spec(NikodraConfig.from_dict(data)))
    cache = CacheManager(model.state_specs(), page_size=16, num_pages=4, num_slots=2, dtype=torch.float32, device="cpu")
    slot = cache.admit("a")
    fixed = list(cache._fixed.values())
    assert any(t.dtype == torch.int32 for t in fixed)
    for t in fixed:
        t[slot].fill_(3)
    cache.release("a")
    again = cache.admit("b")
    assert again == slot and all(float(t[again].abs().sum()) == 0.0 for t in fixed)


def test_pages_before_a_chunk_come_back_and_the_scheduler_counts_on_it():
    from poor_mans_mamba_b200.parts.base import StateSpec
    specs = {0: [("kv", StateSpec.paged("kv", 2, 16, chunk=40))]}
    cache = CacheManager(specs, page_size=16, num_pages=5, num_slots=1, dtype=torch.float32, device="cpu")
    (g,) = cache.groups.values()
    cache.admit("a")
    for pos in range(200):
        cache.grow("a", pos + 1)
        cache.advance("a", 1)
        held = [b for b, p in enumerate(g.tables["a"]) if p >= 0]
        first = (pos + 1) // 40 * 40     # what the next token's chunk starts with
        assert held == list(range(first // 16, pos // 16 + 1)) or (pos + 1 == first and not held)
        cache.check()
    cache.release("a")
    assert g.pool.n_free == 5
    # a prompt longer than the pool is no misfit when its pages come back
    sched = Scheduler(cache, max_batched_tokens=16, max_seqs=1)
    r = sched.add("long", [1] * 300, SamplingParams(max_new_tokens=1))
    while sched.has_work():
        plan = sched.plan()
        for e in plan.entries:
            cache.grow(e.req.id, cache.lengths[e.req.id] + e.count)
            cache.advance(e.req.id, e.count)
        sched.complete(plan, [0 for e in plan.entries if e.samples])
    assert r.status == "done"
    with pytest.raises(ValueError):
        CacheManager({0: [("kv", StateSpec("kv", "paged", planes=2, width=16, window=3, chunk=4))]}, 16, 4, 1, torch.float32, "cpu")


@pytest.mark.parametrize("which", ["A", "B", "C", "M"])
def test_tensor_names_and_shapes_match_the_model_folder(which, tmp_path):
    d, cfg, weights = C.make_model_dir(which, str(tmp_path / which), seed=3)
    assert "decay_rank" not in open(os.path.join(d, "config.json")).read()
    arch, typed = open_model_dir(d)
    model = Model(arch.model_spec(typed))
    specs = model.param_specs()
    want = {k: tuple(v.shape) for k, v in weights.items()}
    first = typed.first_mixing_layer()
    for name in model.ignored_names():     # the first mixing layer has nothing to mix with
        assert name == f"l{first}.mix.vmix" and want.pop(name) == ()
    assert {k: tuple(s.shape) for k, s in specs.items()} == want
    files = ModelFiles(d)
    try:
        assert check_tensors(specs, model.ignored_names(), files, strict=True) == []
    finally:
        files.close()
    kinds = {m for l in model.spec.layers for m in [p.kind for p in l.part("mixers")]}
    assert kinds == {{"attention": "head_norm_attention", "parallel": "normed_parallel", "wkv": "time_mix"}[x["type"]]
                     for x in cfg["layers"]}


def test_random_weights_mode_writes_a_model_that_opens(tmp_path):
    d = write_random_model(C.config("A"), 5, str(tmp_path / "r"))
    arch, typed = open_model_dir(d)
    files = ModelFiles(d)
    try:
        assert check_tensors(Model(arch.model_spec(typed)).param_specs(), [], files, strict=True) == []
    finally:
        files.close()
    assert json.load(open(os.path.join(d, "config.json")))["layers"][2]["mixer"]["decay_rank"] == 5


# ----------------------------------------------------------------------------- frequencies
@pytest.mark.parametrize("dims,base,yarn", [(64, 1e4, (8.0, 256, 32.0, 1.0)), (16, 1000.0, (4.0, 64, 8.0, 1.0)), (32, 1e5, (16.0, 300, 32.0, 1.0)),
                                            (8, 400.0, (2.0, 40, 1.0, 1.0)), (40, 1e6, (3.0, 2e5, 1e4, 0.5)), (2, 3.0, (1.5, 7, 1.0, 0.2))])
def test_scaled_frequencies(dims, base, yarn):
    sc = dict(zip(("factor", "original", "fast", "slow"), yarn))
    got, amp = yarn_frequencies(dims, base, *yarn)
    assert got.dtype == torch.float32 and torch.allclose(got.double(), P.frequencies(dims, base, sc), rtol=1e-7, atol=0.0)
    assert amp == pytest.approx(P.turn_amplitude(sc))


def test_plain_frequencies_by_hand():
    # base 10^4, dims 8: pair i turns 1000 * 10^-i / (2 pi) times within 1,000 positions; pair 1 turns 16 times, pair 3 0.16
    sc = {"factor": 4.0, "original": 1000.0, "fast": 1000 / (2 * math.pi) * 10 ** -0.5, "slow": 1000 / (2 * math.pi) * 10 ** -2.5}
    f = P.frequencies(8, 1e4, sc)     # lo = floor(0.5) = 0, hi = ceil(2.5) = 3
    want = [1.0, 0.1 * (2 / 3 + 1 / 12), 0.01 * (1 / 3 + 2 / 12), 0.001 / 4]
    assert torch.allclose(f, torch.tensor(want, dtype=F64))
    assert P.turn_amplitude(sc) == pytest.approx(0.1 * math.log(4.0) + 1.0) and P.turn_amplitude(None) == 1.0
    assert torch.allclose(P.frequencies(6, 1000.0), torch.tensor([1.0, 0.1, 0.01], dtype=F64))


# ----------------------------------------------------------------------------- the oracle's pieces by hand
def test_plain_bigram_rows_by_hand():
    assert P.bigram_rows([3, 1, 4], 10, 2, 7) == [7, (30 + 2) % 7, (10 + 8) % 7]


def test_plain_rotations_by_hand():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 9.0]]], dtype=F64)
    f, pos = torch.tensor([0.5, 0.1], dtype=F64), torch.tensor([3])
    c, s = [math.cos(1.5), math.cos(0.3)], [math.sin(1.5), math.sin(0.3)]
    halves = [1 * c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + 1 * s[0], 4 * c[1] + 2 * s[1], 9]
    pairs = [1 * c[0] - 2 * s[0], 2 * c[0] + 1 * s[0], 3 * c[1] - 4 * s[1], 4 * c[1] + 3 * s[1], 9]
    assert torch.allclose(P.rotate(x, pos, f, True)[0, 0], torch.tensor(halves, dtype=F64))
    assert torch.allclose(P.rotate(x, pos, f, False)[0, 0], torch.tensor(pairs, dtype=F64))
    double = [2 * v for v in pairs[:4]] + [9]          # the amplitude reaches turned entries only
    assert torch.allclose(P.rotate(x, pos, f, False, 2.0)[0, 0], torch.tensor(double, dtype=F64))


def test_plain_chunks_and_the_one_more_by_hand():
    q = k = torch.zeros(5, 1, 2, dtype=F64)
    v = torch.tensor([1.0, 2.0, 4.0, 8.0, 16.0], dtype=F64).reshape(5, 1, 1)
    out = P.attend_with_one_more(q, k, v, 1.0, P.chunk_mask(5, 3))
    assert torch.allclose(out[:, 0, 0], torch.tensor([1 / 2, 3 / 3, 7 / 4, 8 / 2, 24 / 3], dtype=F64))
    low = torch.full((1, 1, 1), -1.0, dtype=F64)     # a score of -1: the one outweighs it
    out = P.attend_with_one_more(low, -low, torch.ones(1, 1, 1, dtype=F64), 1.0, P.causal_mask(1))
    assert float(out) == pytest.approx(math.exp(-1) / (1 + math.exp(-1)))


def test_plain_retention_and_time_mixing_by_hand():
    q = torch.tensor([[[1.0, 2.0]], [[3.0, 1.0]]], dtype=F64)
    k = torch.tensor([[[1.0, 0.0]], [[0.5, 1.0]]], dtype=F64)
    v = torch.tensor([[[2.0]], [[4.0]]], dtype=F64)
    o = P.retention_scan(q, k, v, [0.5])
    assert torch.allclose(o[:, 0, 0], torch.tensor([2.0, 3 * (1.0 + 2.0) + 1 * 4.0], dtype=F64))
    w = torch.tensor([[[0.5, 0.25]], [[9.0, 9.0]]], dtype=F64)   # the last token's decay is never read
    u = torch.tensor([[10.0, 100.0]], dtype=F64)
    o = P.wkv_scan(q, k, v, w, u)
    # token 0: state zero, only the bonus; token 1: the state holds token 0's write, undecayed
    assert torch.allclose(o[:, 0, 0], torch.tensor([1 * 10 * 1 * 2.0, 3 * 2.0 + 3 * 10 * 0.5 * 4 + 1 * 100 * 1 * 4.0], dtype=F64))
    h = torch.tensor([[1.0], [3.0]], dtype=F64)
    assert torch.allclose(P.shifted_mix(h, torch.tensor([0.25], dtype=F64)), torch.tensor([[0.75], [2.5]], dtype=F64))


def test_plain_gelu_is_the_exact_form():
    z = torch.tensor([-1.0, 0.5, 2.0], dtype=F64)
    assert torch.allclose(P.gelu_erf(z), torch.nn.functional.gelu(z, approximate="none"))


@pytest.mark.parametrize("which", ["A", "B", "C"])
def test_every_tensor_moves_the_plain_logits(which):
    """A tensor that the oracle ignored would hide the same fault in the product."""
    data = C.config(which)
    W = C.make_weights(data, 5)
    toks = C.sequences(data, [9], seed=2)[0]
    base = P.forward(data, W, toks)
    unused = []
    for name in W:
        other = dict(W)
        other[name] = W[name] * 1.5 + 0.25
        if torch.equal(P.forward(data, other, toks), base):
            unused.append(name)
    first = NikodraConfig.from_dict(data).first_mixing_layer()
    assert unused == [f"l{first}.mix.vmix"], unused
