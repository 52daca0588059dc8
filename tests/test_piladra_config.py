"""Piladra's configuration reader, its description as parts, its tensor names, what the cache manager keeps for it, and
the plain implementation's own pieces on cases done by hand (no GPU)."""
import math
import os

import pytest
import torch

import piladra_configs as C
from plain import piladra_plain as P

import poor_mans_mamba_b200.architectures  # noqa: F401  (registration)
from poor_mans_mamba_b200.cache import CacheManager
from poor_mans_mamba_b200.config import ConfigError, resolve_architecture
from poor_mans_mamba_b200.config.piladra import PiladraConfig
from poor_mans_mamba_b200.config.registry import open_model_dir
from poor_mans_mamba_b200.engine.model import Model
from poor_mans_mamba_b200.parts.rope import rotary_frequencies
from poor_mans_mamba_b200.weights.loader import check_tensors
from poor_mans_mamba_b200.weights.safetensors_io import ModelFiles

F64 = torch.float64


@pytest.mark.parametrize("which", ["A", "B", "C", "M"])
def test_every_size_and_constant_is_read(which):
    data = C.config(which)
    cfg = PiladraConfig.from_dict(data)
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.norm_groups) == (
        data["vocab"], data["width"], data["norm"]["eps"], data["norm"]["groups"])
    assert (cfg.canon_taps, cfg.residual_mult, cfg.logit_softcap) == (
        data["canon"]["taps"], data["residual_mult"], data.get("logit_softcap", 0.0))
    if data.get("loop"):
        assert (cfg.loop.start, cfg.loop.stop, cfg.loop.times) == tuple(data["loop"][k] for k in ("start", "stop", "times"))
    else:
        assert cfg.loop is None
    for layer, raw in zip(cfg.layers, data["layers"]):
        m = raw["mixer"]
        assert layer.type == raw["type"]
        assert [x is not None for x in (layer.attention, layer.latent, layer.scan)] == [
            raw["type"] == t for t in ("attention", "latent_attention", "mamba1")]
        if layer.attention is not None:
            x, rot = layer.attention, m.get("rot") or {"dims": 0, "base": 1.0}
            assert (x.heads, x.kv_heads, x.dim, x.vdim, x.scale) == tuple(m[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale"))
            assert (x.rot_dims, x.window) == (rot["dims"], (m.get("mask") or {}).get("size", 0))
            sc = rot.get("scaling")
            assert x.rot_scaling == (None if sc is None else tuple(sc[k] for k in ("factor", "low", "high", "original")))
        elif layer.latent is not None:
            x = layer.latent
            assert (x.heads, x.dim, x.rot_dim, x.vdim, x.kv_rank, x.scale, x.rot_dims, x.rot_base) == (
                m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], m["rot"]["dims"], m["rot"]["base"])
        else:
            x = layer.scan
            assert (x.inner, x.state, x.dt_rank, x.conv) == tuple(m[k] for k in ("inner", "state", "dt_rank", "conv"))
        mlp = raw["mlp"]
        if mlp is None:
            assert layer.dense is None and layer.routed is None
        elif mlp["kind"] == "dense":
            assert layer.dense.ff == mlp["ff"] and layer.routed is None
        else:
            assert (layer.routed.experts, layer.routed.top, layer.routed.expert_ff, layer.routed.shared_ff) == (
                mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"], (mlp.get("shared") or {"ff": 0})["ff"])


def test_the_architecture_is_chosen_by_its_name():
    assert resolve_architecture(C.config("A")).name == "Piladra"


@pytest.mark.parametrize("path,value,needle", [
    (("layers", 0, "mixer", "inner"), 0, "layers[0].mixer.inner"),
    (("layers", 0, "mixer", "dt_rank"), -1, "layers[0].mixer.dt_rank"),
    (("layers", 0, "mixer", "conv"), 0, "layers[0].mixer.conv"),
    (("layers", 1, "mixer", "kv_heads"), 3, "layers[1].mixer.kv_heads"),
    (("layers", 1, "mixer", "rot", "dims"), 7, "layers[1].mixer.rot.dims"),
    (("layers", 1, "mixer", "rot", "dims"), 26, "layers[1].mixer.rot.dims"),
    (("layers", 1, "mixer", "rot", "scaling", "factor"), 0.0, "layers[1].mixer.rot.scaling"),
    (("layers", 1, "mixer", "rot", "scaling", "low"), 9.0, "layers[1].mixer.rot.scaling"),
    (("layers", 1, "mixer", "mask", "size"), -1, "layers[1].mixer.mask.size"),
    (("layers", 2, "mixer", "kv_rank"), 0, "layers[2].mixer.kv_rank"),
    (("layers", 2, "mixer", "rot", "base"), 0.0, "layers[2].mixer.rot.base"),
    (("layers", 0, "mlp", "router", "top"), 7, "layers[0].mlp.router.top"),
    (("layers", 0, "mlp", "shared", "ff"), 0, "layers[0].mlp.shared.ff"),
    (("layers", 1, "mlp", "kind"), "glu", "layers[1].mlp.kind"),
    (("layers", 2, "type"), "mamba2", "layers[2].type"),
    (("norm", "groups"), 5, "norm.groups"),
    (("canon", "taps"), 0, "canon.taps"),
    (("loop", "stop"), 5, "loop"),
    (("loop", "start"), 3, "loop"),
    (("loop", "times"), 0, "loop.times"),
    (("logit_softcap",), -1.0, "logit_softcap"),
    (("width",), 0, "width"),
])
def test_errors_name_the_key(path, value, needle):
    data = C.config("A")
    node = data
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    with pytest.raises(ConfigError) as exc:
        PiladraConfig.from_dict(data)
    assert needle in str(exc.value)


def test_missing_keys_are_refused_and_optional_ones_default():
    for path in (("canon", "taps"), ("norm", "groups"), ("residual_mult",), ("layers", 0, "mixer", "state"),
                 ("layers", 1, "mixer", "scale"), ("layers", 1, "mixer", "vdim"), ("layers", 2, "mixer", "kv_rank"),
                 ("layers", 1, "mixer", "rot", "scaling", "original"), ("loop", "times")):
        data = C.config("A")
        node = data
        for k in path[:-1]:
            node = node[k]
        del node[path[-1]]
        with pytest.raises(ConfigError, match=path[-1]):
            PiladraConfig.from_dict(data)
    data = C.config("A")
    del data["loop"], data["logit_softcap"], data["layers"][0]["mlp"]["shared"], data["layers"][1]["mixer"]["mask"]
    del data["layers"][1]["mixer"]["rot"]["scaling"], data["layers"][3]["mixer"]["rot"]
    data["layers"][1]["mlp"] = None
    cfg = PiladraConfig.from_dict(data)
    assert cfg.loop is None and cfg.logit_softcap == 0.0 and cfg.layers[0].routed.shared_ff == 0
    assert cfg.layers[1].attention.window == 0 and cfg.layers[1].attention.rot_scaling is None
    assert cfg.layers[3].attention.rot_dims == 0 and cfg.layers[1].dense is None


@pytest.mark.parametrize("which", ["A", "B", "C", "M"])
def test_every_run_has_a_cache_of_its_own_and_passes_are_numbered(which):
    data = C.config(which)
    cfg = PiladraConfig.from_dict(data)
    spec = resolve_architecture(data).model_spec(cfg)
    runs = P.layer_runs(data)
    assert [(c.layer, c.pass_index if c.enters else None) for c in spec.order] == runs
    assert [c.cache_of for c in spec.order] == list(range(len(runs)))
    model = Model(spec)
    states = model.state_specs()
    D, taps = data["width"], data["canon"]["taps"]
    for run, (i, _) in enumerate(runs):
        raw, by_name = data["layers"][i], dict(states[run])
        m = raw["mixer"]
        if raw["type"] == "attention":
            kv = by_name["mix.kv"]
            assert kv.window == (m.get("mask") or {}).get("size", 0)
            assert kv.width == m["kv_heads"] * ((max(m["dim"], m["vdim"]) + 15) // 16 * 16)
        elif raw["type"] == "latent_attention":
            kv = by_name["mix.kv"]
            need = m["kv_rank"] + m["rot_dim"]
            assert kv.window == 0 and need <= kv.width < 2 * max(need, 16) and kv.width % 16 == 0
        else:
            assert by_name["mix.S"].shape == (m["inner"], m["state"]) and by_name["mix.S"].dtype == "float32"
            assert by_name["mix.conv"].shape == (m["conv"] - 1, m["inner"])
        for c, there in (("canon1.inputs", taps > 1), ("canon2.inputs", taps > 1 and raw["mlp"] is not None)):
            assert (c in by_name) == there
            if there:
                assert by_name[c].shape == (taps - 1, D) and by_name[c].dtype == "float32"


def test_a_new_request_starts_from_zeros_in_every_run():
    data = C.config("A")
    model = Model(resolve_architecture(data).model_spec(PiladraConfig.from_dict(data)))
    cache = CacheManager(model.state_specs(), page_size=16, num_pages=4, num_slots=2, dtype=torch.float32, device="cpu")
    slot = cache.admit("a")
    fixed = [t for t in cache._fixed.values()]
    for t in fixed:
        t[slot].fill_(3.0)
    cache.release("a")
    again = cache.admit("b")
    assert again == slot and all(float(t[again].abs().sum()) == 0.0 for t in fixed)
    # 8 runs (one layer before the loop, two layers three times, one behind): the last layer has no feed-forward
    assert sum(1 for _, name in cache._fixed if name.startswith("canon")) == 2 * 7 + 1


@pytest.mark.parametrize("which", ["A", "B", "C", "M"])
def test_tensor_names_and_shapes_match_the_model_folder(which, tmp_path):
    d, cfg, weights = C.make_model_dir(which, str(tmp_path / which), seed=3)
    arch, typed = open_model_dir(d)
    model = Model(arch.model_spec(typed))
    specs = model.param_specs()
    assert {k: tuple(s.shape) for k, s in specs.items()} == {k: tuple(v.shape) for k, v in weights.items()}
    files = ModelFiles(os.path.join(d))
    try:
        assert check_tensors(specs, model.ignored_names(), files, strict=True) == []
    finally:
        files.close()


# ----------------------------------------------------------------------------- frequencies
@pytest.mark.parametrize("dims,base,scaling", [(64, 5e5, (8.0, 1.0, 4.0, 8192)), (16, 1000.0, (8.0, 1.0, 4.0, 64)), (40, 1e5, (4.0, 1.0, 3.0, 500)),
                                               (32, 1e4, None), (8, 10.0, (2.0, 2.0, 2.0, 10)), (2, 3.0, (3.0, 0.5, 9.0, 40))])
def test_scaled_frequencies(dims, base, scaling):
    want = P.frequencies(dims, base, None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling)))
    got = rotary_frequencies(dims, base, scaling=scaling)
    assert got.dtype == torch.float32 and torch.allclose(got.double(), want, rtol=1e-7, atol=0.0)


def test_plain_frequencies_by_hand():
    # wavelengths 2 pi, 20 pi, 200 pi against 100 positions: they fit in 15.9, 1.59 and 0.159 times
    f = P.frequencies(6, 1000.0, {"factor": 5.0, "low": 1.0, "high": 4.0, "original": 100})
    n = 100 / (20 * math.pi)
    s = (n - 1.0) / 3.0
    assert torch.allclose(f, torch.tensor([1.0, (1 - s) * 0.1 / 5 + s * 0.1, 0.01 / 5], dtype=F64))
    assert torch.allclose(P.frequencies(6, 1000.0), torch.tensor([1.0, 0.1, 0.01], dtype=F64))


# ----------------------------------------------------------------------------- the oracle's pieces by hand
def test_plain_grouped_norm_and_input_convolution_by_hand():
    x = torch.tensor([[3.0, 4.0, 6.0, 8.0]], dtype=F64)
    w = torch.tensor([1.0, 2.0, 1.0, 0.5], dtype=F64)
    a, b = math.sqrt(12.5 + 1.0), math.sqrt(50.0 + 1.0)
    assert torch.allclose(P.grouped_norm(x, w, 1.0, 2), torch.tensor([[3 / a, 8 / a, 6 / b, 4 / b]], dtype=F64))
    h = torch.tensor([[1.0], [2.0], [4.0]], dtype=F64)
    taps = torch.tensor([[10.0, 0.1, 1.0]], dtype=F64)   # two back, one back, now
    assert torch.allclose(P.input_conv(h, taps), torch.tensor([[2.0], [4.0 + 0.1], [8.0 + 0.2 + 10.0]], dtype=F64))


def test_plain_selective_scan_by_hand():
    x, dt = torch.tensor([[2.0], [1.0]], dtype=F64), torch.tensor([[0.5], [1.0]], dtype=F64)
    A, B, Cm = torch.tensor([[-1.0, -2.0]], dtype=F64), torch.tensor([[1.0, 3.0], [0.0, 1.0]], dtype=F64), torch.tensor([[1.0, 1.0], [2.0, 0.5]], dtype=F64)
    y = P.selective_scan(x, dt, A, B, Cm, torch.tensor([0.25], dtype=F64))
    s1 = [1.0, 3.0]
    s2 = [math.exp(-1.0) * 1.0, math.exp(-2.0) * 3.0 + 1.0]
    assert torch.allclose(y[:, 0], torch.tensor([s1[0] + s1[1] + 0.5, 2 * s2[0] + 0.5 * s2[1] + 0.25], dtype=F64))


def test_plain_router_and_weighted_input_by_hand():
    z = torch.tensor([0.0, 2.0, -1.0, 2.0], dtype=F64)
    chosen, ws = P.route(z, 3)
    assert chosen == [1, 3, 0]
    assert torch.allclose(torch.stack(ws), torch.sigmoid(torch.tensor([2.0, 2.0, 0.0], dtype=F64)))   # they need not sum to one
    W = {"m.router": torch.tensor([[1.0]], dtype=F64)}
    for n, v in (("gate", 3.0), ("up", 2.0), ("down", 1.0)):
        W[f"m.e0.{n}"] = torch.tensor([[v]], dtype=F64)
    out = P.routed_ffn(torch.tensor([[1.5]], dtype=F64), W, "m.", {"router": {"top": 1}})
    u = 1.5 / (1 + math.exp(-1.5))                       # the weighted input
    assert float(out) == pytest.approx(3 * u / (1 + math.exp(-3 * u)) * 2 * u)


def test_plain_sink_window_and_softcap_by_hand():
    q = k = torch.zeros(3, 1, 2, dtype=F64)
    v = torch.tensor([1.0, 2.0, 4.0], dtype=F64).reshape(3, 1, 1)
    out = P.masked_softmax_attention(q, k, v, 1.0, P.window_mask(3, 2), torch.tensor([math.log(2.0)], dtype=F64))
    assert torch.allclose(out[:, 0, 0], torch.tensor([1 / 3, 3 / 4, 6 / 4], dtype=F64))   # the sink counts as two keys
    data = C.config("C")
    W = C.make_weights(data, 1)
    toks = C.sequences(data, [6])[0]
    plain = P.forward(data, W, toks)
    assert torch.allclose(P.forward(dict(data, logit_softcap=3.0), W, toks), 3.0 * torch.tanh(plain / 3.0))


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
    # only experts that no token of this short sequence chose may be without effect
    assert all(".mlp.e" in n for n in unused), unused


def test_a_pass_vector_counts_for_its_own_pass_only():
    data = C.config("A")
    W = C.make_weights(data, 5)
    toks = C.sequences(data, [7])[0]
    runs = P.layer_runs(data)
    base = []
    P.forward(data, W, toks, layers_out=base)
    for t in range(data["loop"]["times"]):
        other = dict(W)
        other["loop.step"] = W["loop.step"].clone()
        other["loop.step"][t] += 1.0
        got = []
        P.forward(data, other, toks, layers_out=got)
        first = next(r for r, (_, begins) in enumerate(runs) if begins == t)
        assert all(torch.equal(a, b) for a, b in zip(base[:first], got[:first])) and not torch.equal(base[first], got[first])


def test_decisive_routers_leave_no_close_call():
    for which in ("A", "B", "C"):
        data = C.config(which)
        W = C.make_weights(data, 7)
        C.decisive_routers(W)
        gaps = []
        routed = P.routed_ffn

        def spy(x, W, pre, mlp):
            s = torch.sigmoid(P.linear(x, W[pre + "router"])).sort(dim=-1, descending=True).values
            if mlp["router"]["top"] < s.shape[1]:
                z = torch.logit(s)
                gaps.append(float((z[:, mlp["router"]["top"] - 1] - z[:, mlp["router"]["top"]]).min()))
            return routed(x, W, pre, mlp)
        P.routed_ffn = spy
        try:
            P.forward(data, W, C.sequences(data, [40])[0])
        finally:
            P.routed_ffn = routed
        assert gaps and min(gaps) > 0.05, (which, gaps)
