"""Nikodra through the engine against the plain implementation (GPU): every way of cutting the work, tiny
configurations that differ in every size and option, float32 and bfloat16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import gpu_harness as H
import nikodra_configs as C
from plain import nikodra_plain as P

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_FRAC = 3e-5
LENGTHS = (1, 2, 9, 40, 77, 131, 203)
DTYPES = ("float32", "bfloat16")


def check_rows(got, ref, dtype, what, f32_frac=F32_FRAC, bf16_frac=H.BF16_FRAC):
    if dtype == "float32":
        return H.check_rows(got, ref, dtype, what, f32_frac=f32_frac)
    got = got.detach().double().cpu()
    assert got.shape == ref.shape and bool(torch.isfinite(got).all()), what
    frac = (got - ref).abs().max(dim=1).values / float(ref.abs().max())
    assert float(frac.max()) <= bf16_frac, f"{what}: {float(frac.max()):.4f} > {bf16_frac:.4f} at row {int(frac.argmax())}"


def rounding_noise(cfg, weights, seqs, refs):
    """How far the plain logits move (as a fraction of the largest one) when every matrix product's operand and result
    are rounded to bfloat16.  A head whose result is close to zero is divided by its own root mean square, so that a
    few positions of a few models magnify rounding to several per cent."""
    exact = P.linear

    def rounded(x, w, b=None):
        y = exact(x.to(torch.bfloat16).double(), w).to(torch.bfloat16).double()
        return y if b is None else y + b
    P.linear = rounded
    try:
        return max(float((P.forward(cfg, weights, s, torch.float64) - r).abs().max() / r.abs().max()) for s, r in zip(seqs, refs))
    finally:
        P.linear = exact


class Case:
    def __init__(self, which, tmp, lengths=LENGTHS, seq_seed=7, seed=None, edit=None, patch=None):
        self.which = which if isinstance(which, str) else "custom"
        seed = ord(self.which[0]) if seed is None else seed
        self.dir, self.cfg, self.weights = C.make_model_dir(which, str(tmp), seed=seed, edit=edit, patch=patch)
        self.seqs = C.sequences(self.cfg, lengths, seed=seq_seed)
        self.refs = [P.forward(self.cfg, self.weights, s, torch.float64) for s in self.seqs]
        self.bf16_frac = max(H.BF16_FRAC, 3.0 * rounding_noise(self.cfg, self.weights, self.seqs, self.refs))

    def check(self, script, dtype, what, page_size=16, num_pages=40, num_slots=4, f32_frac=F32_FRAC, only=None):
        runner = H.make_runner(self.dir, dtype, page_size=page_size, num_pages=num_pages, num_slots=num_slots)
        out = H.run_script(runner, self.seqs, script)
        runner.check_kernels(wait=True)
        for i, ref in enumerate(self.refs):
            if only is None or i in only:
                check_rows(out[i], ref, dtype, f"{self.which} {dtype} {what} seq {i} (len {len(self.seqs[i])})", f32_frac=f32_frac,
                           bf16_frac=self.bf16_frac)
        return runner


@pytest.fixture(scope="module", params=["A", "B", "C"])
def case(request, tmp_path_factory):
    return Case(request.param, tmp_path_factory.mktemp(f"nk{request.param}"))


def test_the_stream_after_every_layer(case):
    """The float32 residual stream after every layer against the plain implementation: the first difference names it."""
    seq, want, got = case.seqs[4], [], []
    P.forward(case.cfg, case.weights, seq, torch.float64, layers_out=want)
    runner = H.make_runner(case.dir, "float32", page_size=16, num_pages=8, num_slots=1)
    for layer in runner.model.layers:
        def forward(stream, ctx, cache, orig=layer.forward):
            orig(stream, ctx, cache)
            got.append(stream.flush().clone())
        layer.forward = forward
    H.run_script(runner, [seq], H.script_whole([seq]))
    assert len(got) == len(want) == len(case.cfg["layers"])
    for i, (g, w) in enumerate(zip(got, want)):
        err = float((g.double().cpu() - w).abs().max())
        assert err <= 2e-5 * max(1.0, float(w.abs().max())), f"{case.which}: stream after layer {i}: {err:.3e}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cutting", ["whole", "tail", "portions", "mixed"])
def test_cuttings_agree_with_plain(case, dtype, cutting):
    seqs, page_size = case.seqs, 16
    if cutting == "mixed":
        # so few pages and slots that they are used again
        budget = max((len(s) + page_size - 1) // page_size for s in seqs) + 5
        script = H.script_mixed(seqs, max_live=3, seed=5, budget_pages=budget, page_size=page_size)
        assert any(len(p) > 1 and any(n == 1 for _, _, n in p) and any(n > 1 for _, _, n in p) for p, _ in script)
        runner = case.check(script, dtype, cutting, num_pages=budget, num_slots=3)
    else:
        script = {"whole": H.script_whole, "portions": H.script_portions,
                  "tail": lambda s: H.script_tail_one_by_one(s, tail=70)}[cutting](seqs)
        runner = case.check(script, dtype, cutting, num_pages=16, num_slots=2)
    for g in runner.cache.groups.values():
        assert g.pool.n_free == g.num_pages  # every page came back
    assert runner.cache.free_slots == runner.cache.num_slots


@pytest.mark.parametrize("page_size", [16, 64])
def test_portions_of_two_and_three_tokens(case, page_size):
    """Both parities of every page's and chunk's edge are met."""
    i, n = 5, len(case.seqs[5])
    for width in (2, 3):
        script = [([(i, a, min(width, n - a))], [i] if a + width >= n else []) for a in range(0, n, width)]
        case.check(script, "float32", f"portions of {width}", page_size=page_size, num_pages=max(4, 256 // page_size), num_slots=1, only=[i])


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_from_the_first_token(case, dtype):
    """One prompt token, then 202 tokens one by one: chunks pass over decoded tokens, the states start from nothing."""
    n = len(case.seqs[6])
    case.check([([(6, p, 1)], [6] if p == n - 1 else []) for p in range(n)], dtype, "long decoding", num_slots=1, num_pages=16, only=[6])


@pytest.mark.parametrize("dtype", DTYPES)
def test_batch_of_unequal_requests_equals_each_alone(case, dtype):
    seqs, pick = case.seqs, [1, 3, 4, 6]
    half = {i: len(seqs[i]) // 2 for i in pick}
    case.check([([(i, 0, half[i]) for i in pick], []), ([(i, half[i], len(seqs[i]) - half[i]) for i in pick], pick)], dtype, "batched", only=pick)


def test_slot_and_pages_used_again_start_clean(case):
    """A request that takes the slot and pages of a finished one sees nothing of it: neither its keys nor its states nor
    its last token."""
    case.check([([(6, 0, 203)], [6]), ([(5, 0, 50)], []), ([(5, 50, 81)], [5]), ([(3, 0, 1)], []), ([(3, 1, 39)], [3])], "float32", "reuse",
               num_pages=13, num_slots=1, only=[6, 5, 3])


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_request_sits_out_while_others_run(case, dtype):
    script = [([(5, 0, 1), (3, 0, 2)], []), ([(5, 1, 1), (3, 2, 38)], [3]), ([(4, 0, 77)], []), ([(2, 0, 9), (5, 2, 2)], [2]),
              ([(1, 0, 1)], []), ([(1, 1, 1), (5, 4, 70)], [1]), ([(5, 74, 57)], [5, 4])]
    case.check(script, dtype, "sits out", num_pages=30, num_slots=3, only=[5, 3, 4, 2, 1])


def test_pages_before_a_chunk_come_back(tmp_path):
    """A pool far smaller than the request is enough for a model whose attention all stays within chunks."""
    def patch(cfg):
        cfg["layers"] = [l for l in cfg["layers"] if l["type"] != "attention"]
    case = Case("A", tmp_path, lengths=(400,), seq_seed=5, seed=17, patch=patch)
    runner = H.make_runner(case.dir, "float32", page_size=16, num_pages=9, num_slots=1)
    held = []
    orig = runner.cache.advance

    def advance(req, n):
        out = orig(req, n)
        held.append(max(sum(1 for p in g.tables[req] if p >= 0) for g in runner.cache.groups.values()))
        return out
    runner.cache.advance = advance
    script = [([(0, 0, 100)], [])] + [([(0, p, min(7, 400 - p))], [0] if p + 7 >= 400 else []) for p in range(100, 400, 7)]
    out = H.run_script(runner, case.seqs, script)
    check_rows(out[0], case.refs[0], "float32", "pages given back")
    assert [g.chunk for g in runner.cache.groups.values()] == [24] and max(held[1:]) <= 3


def _loud(cfg):
    """Weights under which a lost key, a chunk that is one token off, a missing one in the denominator, a wrong angle, an
    unscaled frequency, a lost state, a wrong previous token or unmixed values cannot hide: the query and key norms
    have one large unturned (or slowest turning) entry, the low-rank decays forget slowly, the bigram rows are large."""
    def edit(W):
        for i, l in enumerate(cfg["layers"]):
            p = f"l{i}.mix."
            if l["type"] == "attention":
                W[p + "q.norm"][-1] *= 2.5
                W[p + "k.norm"][-1] *= 2.5
            elif l["type"] == "parallel":
                W[p + "left.q"][::l["mixer"]["left"]["dim"]] *= 2.0
                W[p + "left.k"][::l["mixer"]["left"]["dim"]] *= 2.0
            else:
                W[p + "w0"] -= 1.0
                W[p + "w2"] *= 2.5
        if "bigram" in W:
            W["bigram"] *= 1.3
    return edit


@pytest.mark.parametrize("which", ["A", "B"])
def test_loud_far_keys_chunks_positions_and_states(which, tmp_path):
    def patch(cfg):
        for l in cfg["layers"]:
            if l["type"] == "parallel":
                l["mixer"]["left"]["scale"] *= 3.0
    case = Case(which, tmp_path, lengths=(300,), seq_seed=3, seed=12, edit=_loud(C.CONFIGS[which]), patch=patch)
    ref, toks = case.refs[0], case.seqs[0]

    # the oracle itself: with a mechanism a little off the logits move visibly
    def moved(change=None, swap=None):
        cfg, W = json.loads(json.dumps(case.cfg)), {k: v.clone() for k, v in case.weights.items()}
        if change:
            change(cfg, W)
        saved = {}
        for name, fn in (swap or {}).items():
            saved[name] = getattr(P, name)
            setattr(P, name, fn)
        try:
            return float((P.forward(cfg, W, toks, torch.float64) - ref).abs().max()) / float(ref.abs().max())
        finally:
            for name, fn in saved.items():
                setattr(P, name, fn)

    def chunk_by(delta):
        def change(cfg, W):
            for l in cfg["layers"]:
                if l["type"] == "parallel":
                    l["mixer"]["left"]["mask"]["size"] += delta
        return change

    def unscaled(cfg, W):
        for l in cfg["layers"]:
            l["mixer"].get("rot", {}).pop("scaling", None)

    def unmixed(cfg, W):
        for k in W:
            if k.endswith("vmix"):
                W[k] = W[k] * 0.0

    def tanh_is_lost(cfg, W):
        for k in W:
            if k.endswith("mix.w2"):
                W[k] = W[k] * 0.0

    def no_bonus(cfg, W):
        for k in W:
            if k.endswith("mix.u"):
                W[k] = W[k] * 0.0

    def bigram_swapped(cfg, W):
        b = cfg["embedding"]["bigram"]
        b["mul_prev"], b["mul_cur"] = b["mul_cur"], b["mul_prev"]

    def plain_softmax(q, k, v, scale, mask):
        T, Hq, _ = q.shape
        rep = Hq // k.shape[1]
        s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, 1)) * scale
        p = torch.softmax(s.masked_fill(~mask, -float("inf")), dim=-1)
        return torch.einsum("hij,jhd->ihd", p, v.repeat_interleave(rep, 1))
    for change in (chunk_by(1), chunk_by(-1), unscaled, unmixed, tanh_is_lost, no_bonus, bigram_swapped):
        assert moved(change) > 3 * H.BF16_FRAC, change
    assert moved(swap={"attend_with_one_more": plain_softmax}) > 3 * H.BF16_FRAC
    assert moved(swap={"turn_amplitude": lambda s: 1.0}) > 1.5 * H.BF16_FRAC
    for dtype in DTYPES:
        for script in (H.script_whole(case.seqs), H.script_tail_one_by_one(case.seqs, tail=100), H.script_portions(case.seqs, seed=2)):
            runner = H.make_runner(case.dir, dtype, page_size=16, num_pages=24, num_slots=1)
            out = H.run_script(runner, case.seqs, script)
            if dtype == "float32":
                check_rows(out[0], ref, dtype, f"loud {which}", f32_frac=6e-5)
                continue
            # loud scores magnify bfloat16 rounding at a few positions: all rows within twice the usual bound or three
            # times what rounding alone does, all but one in fifty within the usual bound
            frac = (out[0].double() - ref).abs().max(dim=1).values / float(ref.abs().max())
            assert bool(torch.isfinite(out[0]).all()) and float(frac.max()) <= max(2 * H.BF16_FRAC, case.bf16_frac), f"loud {which}: {float(frac.max()):.3f}"
            assert int((frac > H.BF16_FRAC).sum()) <= len(frac) // 50


def test_options_that_one_model_leaves_equal(tmp_path):
    """Equal sizes everywhere, one head, a chunk of one token, no feed-forwards, a residual multiplier of one, a single
    bucket, no rotation."""
    cfg = {"architecture": "Nikodra", "vocab": 64, "width": 64, "norm": {"eps": 1e-5}, "residual_mult": 1.0,
           "embedding": {"bigram": {"buckets": 1, "mul_prev": 1, "mul_cur": 1}}, "layers": [
        C.layer(C.attention(1, 1, 16, 16, 1.0), None), C.layer(C.parallel((1, 1, 16, 16, 1.0, 1), (16, 16, (1.0,), None)), None),
        C.layer(C.wkv(1, 16, 16), None), C.layer(C.attention(1, 1, 16, 16, 1.0, rot=(16, 2.0), yarn=(1.0, 16, 1.0, 1.0)), None)]}
    case = Case(cfg, tmp_path, lengths=(57, 18), seed=31)
    for dtype in DTYPES:
        for name, script in (("whole", H.script_whole(case.seqs)), ("portions", H.script_portions(case.seqs, seed=4)),
                             ("tail", H.script_tail_one_by_one(case.seqs, tail=30))):
            case.check(script, dtype, name, num_pages=8, num_slots=1)


def test_sizes_that_are_multiples_of_nothing(tmp_path):
    """A width that is no multiple of 4, head sizes that are no multiples of 4, an odd vocabulary: the scalar forms of the
    kernels, recurrences token by token and the float products."""
    cfg = {"architecture": "Nikodra", "vocab": 77, "width": 50, "norm": {"eps": 1e-5}, "residual_mult": 0.4,
           "embedding": {"bigram": {"buckets": 13, "mul_prev": 7, "mul_cur": 5}}, "layers": [
        C.layer(C.attention(3, 3, 10, 13, 0.3, rot=(6, 40.0), yarn=(3.0, 30, 2.0, 0.5)), 33),
        C.layer(C.parallel((3, 1, 9, 11, 0.4, 7), (10, 7, (0.9, 0.5, 0.99), (6, 30.0))), 41),
        C.layer(C.wkv(3, 11, 7), 27), C.layer(C.attention(3, 3, 6, 13, 0.3, rot=(2, 9.0)), 19)]}
    case = Case(cfg, tmp_path, lengths=(65, 3), seed=15)
    for dtype in DTYPES:
        for name, script in (("whole", H.script_whole(case.seqs)), ("portions", H.script_portions(case.seqs, seed=6)),
                             ("tail", H.script_tail_one_by_one(case.seqs, tail=25))):
            case.check(script, dtype, name, num_pages=8, num_slots=1)


def test_greedy_generation_through_the_engine(case):
    """Engine.generate (scheduler, sampler, decode graphs) against greedy decoding with the plain implementation,
    float32; bfloat16 with graphs against bfloat16 step by step."""
    from poor_mans_mamba_b200.entry import Engine
    prompts, n_new = [case.seqs[2], case.seqs[3][:23], case.seqs[1]], 12
    eng = Engine(case.dir, dtype="float32", max_tokens=1024, max_seqs=4, page_size=16, max_batched_tokens=32)
    got = eng.generate(prompts, max_new_tokens=n_new, eos_token_id=-1)
    for p, g in zip(prompts, got):
        toks = list(p)
        for _ in range(n_new):
            lg = P.forward(case.cfg, case.weights, toks, torch.float64)[-1]
            top2 = torch.topk(lg, 2).values
            if float(top2[0] - top2[1]) < 1e-3:
                break  # a near tie: the two may disagree from here on without either being wrong
            toks.append(int(lg.argmax()))
        want = toks[len(p):]
        assert g[:len(want)] == want
    a, b = (Engine(case.dir, dtype="bfloat16", max_tokens=1024, max_seqs=4, page_size=16, cuda_graphs=graphs).generate(
        prompts, max_new_tokens=n_new, eos_token_id=-1) for graphs in (True, False))
    assert a == b


def test_replayed_prompt_steps_are_what_issued_ones_are(case):
    """The same cut three times through one engine: issued, recorded, replayed; then decoding on from it."""
    from poor_mans_mamba_b200.entry import Engine
    eng = Engine(case.dir, dtype="bfloat16", max_tokens=1024, max_seqs=2, page_size=16)
    outs = [eng.generate([case.seqs[4]], max_new_tokens=9, eos_token_id=-1)[0] for _ in range(4)]
    assert all(o == outs[0] for o in outs)


def test_trace_program_replays_a_schedule(case, tmp_path):
    if case.which != "A":
        pytest.skip("one configuration is enough for the program")
    seqs, refs, V = case.seqs, case.refs, case.cfg["vocab"]
    steps = [
        {"step": 0, "entries": [{"id": "x", "tokens": seqs[3][:17], "want": [0, 16]}, {"id": "y", "tokens": seqs[2], "want": [8]}], "end": ["y"]},
        {"step": 1, "entries": [{"id": "x", "tokens": seqs[3][17:19], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "x", "tokens": seqs[3][19:], "want": [len(seqs[3]) - 20]}, {"id": "z", "tokens": seqs[1], "want": [1]}],
         "end": ["x", "z"]},
    ]
    for dtype in DTYPES:
        out_dir = str(tmp_path / f"out_{dtype}")
        proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", case.dir, "--dtype", dtype,
                               "--out", out_dir, "--max-tokens", "128"],
                              input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        s0, s2 = (torch.from_numpy(np.fromfile(os.path.join(out_dir, f), dtype="<f4").reshape(-1, V)) for f in ("0.f32", "2.f32"))
        assert not os.path.exists(os.path.join(out_dir, "1.f32"))
        check_rows(s0, torch.stack([refs[3][0], refs[3][16], refs[2][8]]), dtype, "trace step 0")
        check_rows(s2, torch.stack([refs[3][-1], refs[1][1]]), dtype, "trace step 2")


def test_command_line_generates_from_a_model_folder(case):
    if case.which != "B":
        pytest.skip("one configuration is enough for the program")
    prompt = ",".join(str(t) for t in case.seqs[2])
    proc = subprocess.run([sys.executable, "-m", "poor_mans_mamba_b200", case.dir, "64", "GPU", "1", "2", "5", "--dtype", "float32",
                           "--prompt-ids", prompt, "--page-size", "16"], capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert proc.returncode == 0, proc.stderr[-2000:]
    lines = [l for l in proc.stdout.splitlines() if l.startswith("req_id=")]
    assert len(lines) == 2 and all("gen_tokens=5" in l for l in lines)
    toks = list(case.seqs[2])
    for _ in range(5):
        toks.append(int(P.forward(case.cfg, case.weights, toks, torch.float64)[-1].argmax()))
    assert str(toks[len(case.seqs[2]):]) in lines[0]


def test_medium_sizes_where_the_tensor_core_forms_run(tmp_path):
    """Heads of 64 and 128 entries, prompts long enough for the tcgen05 attention and for recurrences in chunks, pages of
    64 tokens: whole, in portions that cut pages and chunks anywhere, and with a long tail decoded."""
    case = Case("M", tmp_path, lengths=(700, 333), seq_seed=9, seed=21)
    for dtype in DTYPES:
        for name, script in (("whole", H.script_whole(case.seqs)), ("tail", H.script_tail_one_by_one(case.seqs, tail=120)),
                             ("portions", [([(0, 0, 257)], []), ([(0, 257, 2), (1, 0, 130)], []), ([(0, 259, 300), (1, 130, 1)], []),
                                           ([(0, 559, 141), (1, 131, 202)], [0, 1])])):
            case.check(script, dtype, name, page_size=64, num_pages=20, num_slots=2, f32_frac=6e-5)


def _random_config(seed):
    """A configuration drawn at random from the ranges a small model of this design may take."""
    import random
    rng = random.Random(7000 + seed)
    width = rng.choice([96, 136, 160, 200, 264, 328])
    layers, mixing = [], (rng.choice([1, 2, 3]), rng.choice([8, 16, 40, 64]))
    for i in range(rng.randint(3, 6)):
        kind = rng.choice(["attention", "parallel", "wkv"])
        if kind == "attention":
            v_mix = rng.random() < 0.7
            G, dv = mixing if v_mix else (rng.choice([1, 2, 3]), rng.choice([8, 16, 24, 48]))
            dim = rng.choice([8, 16, 24, 32, 64, 128])
            rot = (rng.choice([dim, dim, dim // 2]), rng.choice([100.0, 1e4, 1e6])) if rng.random() < 0.9 else None
            yarn = (rng.choice([2.0, 8.0, 40.0]), rng.choice([32, 128, 4096]), rng.choice([4.0, 32.0]), rng.choice([0.5, 1.0])) if rng.random() < 0.7 else None
            mixer = C.attention(G * rng.randint(1, 6), G, dim, dv, dim ** -0.5, rot=rot, yarn=yarn if rot else None, v_mix=v_mix)
        elif kind == "parallel":
            G, dim, rd = rng.choice([1, 2, 3]), rng.choice([8, 16, 48, 64, 96]), rng.choice([8, 16, 32, 64, 96])
            decays = [rng.choice([0.5, 0.9, 0.97, 0.99, 0.998]) for _ in range(rng.randint(1, 6))]
            mixer = C.parallel((G * rng.randint(1, 4), G, dim, rng.choice([dim, 16, 40]), dim ** -0.5, rng.choice([1, 7, 16, 40, 64, 100])),
                               (rd, rng.choice([rd, 16, 48]), decays, (rng.choice([rd, rd // 2]), rng.choice([100.0, 1e6]))))
        else:
            mixer = C.wkv(rng.randint(1, 6), rng.choice([8, 16, 32, 64]), rng.choice([4, 8, 13, 16, 32]))
        layers.append(C.layer(mixer, None if rng.random() < 0.2 else 8 * rng.randint(8, 60)))
    cfg = {"architecture": "Nikodra", "vocab": rng.randint(100, 700), "width": width, "norm": {"eps": rng.choice([1e-6, 1e-5])},
           "residual_mult": rng.choice([0.2, 0.5, 1.0]), "layers": layers}
    if rng.random() < 0.9:
        cfg["embedding"] = {"bigram": {"buckets": rng.randint(2, 900), "mul_prev": rng.randint(1, 5000), "mul_cur": rng.randint(1, 5000)}}
    return cfg


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(seed, tmp_path):
    cfg = _random_config(seed)
    case = Case(cfg, tmp_path, lengths=(150, 37, 70), seq_seed=seed, seed=50 + seed)
    for dtype in DTYPES:
        for name, script in (("whole", H.script_whole(case.seqs)),
                             ("mixed", H.script_mixed(case.seqs, max_live=3, seed=seed, budget_pages=8, page_size=64))):
            case.check(script, dtype, f"random {seed} {name} {json.dumps(cfg)[:200]}", page_size=64, num_pages=8, num_slots=3, f32_frac=6e-5)
