"""Each mechanism of the Piladra parts alone against its plain function (GPU): the kernels are called as the model
calls them, on inputs made so that a fault shows."""
import math

import pytest
import torch

from plain import piladra_plain as P

from poor_mans_mamba_b200.engine.workspace import Workspace
from poor_mans_mamba_b200.kernels import ops as K
from poor_mans_mamba_b200.parts.base import LayerCache, PartSpec, build_part
from poor_mans_mamba_b200.parts.block import ResidualStream
import poor_mans_mamba_b200.parts  # noqa: F401  (registration)

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def rnd(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(torch.bfloat16).float()


def close(got, want, dtype, what, f32=2e-5, bf16=2e-2):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} vs {tuple(want.shape)}"
    tol = (f32 if dtype == torch.float32 else bf16) * max(1.0, float(want.abs().max()))
    err = float((got - want).abs().max())
    assert err <= tol, f"{what}: {err:.3e} > {tol:.3e}"


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


class Ctx:
    """What the parts read of a step: sequences of the given lengths, one after the other, in the given slots."""

    def __init__(self, lens, slots, dtype):
        self.dtype, self.workspace = dtype, Workspace(torch.device(DEV))
        self.new_lens, self.n_seq, self.n_tokens = list(lens), len(lens), sum(lens)
        self.decode_only = all(n == 1 for n in lens)
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        self.cu_seqlens, self.slots = i32(cu), i32(slots)
        self.seq_of = i32([s for s, n in enumerate(lens) for _ in range(n)])


# ----------------------------------------------------------------------------- fold, grouped norm, input convolution
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,groups", [(44, 1), (72, 3), (100, 5), (50, 25), (1024, 8), (3072, 2), (5000, 4), (96, 96)])
def test_norm_over_groups_with_branches_and_a_vector(dtype, D, groups):
    T, eps = 9, 1e-2
    h0, vec, w = rnd(T, D, seed=1, scale=2.0), rnd(D, seed=3), rnd(D, seed=8) * 0.2 + 1.0
    h0[:, :D // groups] *= 20.0  # one group much larger than the others: the whole row's root mean square would show
    bs = [(rnd(T, D, seed=2), 0.7), (rnd(T, D, seed=4), -1.5)]
    for n_b, with_vec in ((0, False), (1, True), (2, True), (2, False)):
        dev_b = [(b.to(DEV, dtype), s) for b, s in bs[:n_b]]
        x = h0.double() + sum((s * b.to(dtype).double() for b, s in bs[:n_b]), torch.zeros(T, D, dtype=torch.float64))
        x = x + (vec.double() if with_vec else 0.0)
        want = P.grouped_norm(x, w.double(), eps, groups)
        h, out = h0.to(DEV).clone(), torch.empty(T, D, dtype=dtype, device=DEV)
        K.fold_norm(h, h, dev_b, vec.to(DEV) if with_vec else None, w.to(DEV), eps, groups, out)
        close(h, x, torch.float32, "stream")
        close(out, want, dtype, "normed stream", bf16=1e-2)
        rows = [7, 0, 3]
        h, out = h0.to(DEV).clone(), torch.empty(len(rows), D, dtype=dtype, device=DEV)
        K.fold_norm(h, h, dev_b, vec.to(DEV) if with_vec else None, w.to(DEV), eps, groups, out, i32(rows))
        assert torch.equal(h.cpu(), h0)
        close(out, want[rows], dtype, "chosen rows", bf16=1e-2)
        if n_b or with_vec:
            h = h0.to(DEV).clone()
            K.fold_norm(h, h, dev_b, vec.to(DEV) if with_vec else None, None, 0.0, 1, None)
            close(h, x, torch.float32, "fold alone")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
@pytest.mark.parametrize("D,groups", [(50, 2), (96, 3), (1024, 2)])
def test_input_convolution_in_any_cut(dtype, taps, D, groups):
    """Three requests through steps whose portions have 1 to 40 tokens (shorter and longer than the convolution, single
    tokens beside long portions, steps of single tokens only), branches folded in on the way: the outputs, the folded
    stream and the windows are what the whole sequences give."""
    eps, L = 1e-3, taps - 1
    lengths = [61, 47, 23]
    cuts = [[1, 2, 40, 1, 9, 8], [5, 1, 1, 39, 1, 0], [0, 20, 1, 1, 1, 0]]
    assert [sum(c) for c in cuts] == lengths
    h = [rnd(n, D, seed=i, scale=1.5) for i, n in enumerate(lengths)]
    b = [rnd(n, D, seed=10 + i).to(dtype).float() for i, n in enumerate(lengths)]
    vec, w, ker = rnd(D, seed=20), rnd(D, seed=21) * 0.2 + 1.0, rnd(D, taps, seed=22, scale=0.6)
    x = [hh.double() + 0.6 * bb.double() + vec.double() for hh, bb in zip(h, b)]
    normed = [P.grouped_norm(v, w.double(), eps, groups) for v in x]
    want = [P.input_conv(n, ker.double()) for n in normed]
    window = torch.full((5, L, D), 7.0, dtype=torch.float32, device=DEV)   # slots used before
    slots = [3, 0, 2]
    window[slots] = 0.0
    ker_t = ker.t().contiguous().to(DEV)
    at = [0, 0, 0]
    for step in range(len(cuts[0])):
        live = [s for s in range(3) if cuts[s][step] > 0]
        lens = [cuts[s][step] for s in live]
        T = sum(lens)
        ctx = Ctx(lens, [slots[s] for s in live], dtype)
        hh = torch.cat([h[s][at[s]:at[s] + n] for s, n in zip(live, lens)]).to(DEV)
        bb = torch.cat([b[s][at[s]:at[s] + n] for s, n in zip(live, lens)]).to(DEV, dtype)
        before = hh.clone()
        dst = hh if ctx.decode_only else torch.full_like(hh, 9.0)
        out = torch.empty(T, D, dtype=dtype, device=DEV)
        K.fold_norm(hh, dst, [(bb, 0.6)], vec.to(DEV), w.to(DEV), eps, groups, out, conv=ker_t, window=window if L else None,
                    cu=ctx.cu_seqlens, slots=ctx.slots, seq_of=ctx.seq_of, n_seq=ctx.n_seq, one_token=ctx.decode_only)
        if dst is not hh:
            assert torch.equal(hh, before)
        r = 0
        for s, n in zip(live, lens):
            close(dst[r:r + n], x[s][at[s]:at[s] + n], torch.float32, f"stream, step {step}")
            close(out[r:r + n], want[s][at[s]:at[s] + n], dtype, f"taps {taps} step {step} sequence {s}", bf16=1e-2)
            r += n
            at[s] += n
            for k in range(L):   # oldest first; zeros before the sequence's start
                p = at[s] - L + k
                row = normed[s][p] if p >= 0 else torch.zeros(D, dtype=torch.float64)
                close(window[slots[s], k], row, torch.float32, "window")
    assert torch.equal(window[[1, 4]], torch.full_like(window[[1, 4]], 7.0))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 3, 6])
def test_input_map_behind_a_norm_of_another_kind_runs_on_its_own(dtype, taps):
    """The same part behind the statistic-free norm: the convolution is a launch of its own over the stored rows, and a
    waiting vector is folded first."""
    D, lens = 40, [13, 1, 6]
    part = build_part("input_map", PartSpec("residual_conv", "c", {"taps": taps}), hidden_size=D)
    ker = rnd(D, taps, seed=1, scale=0.6)
    part.bind({"": ker.to(DEV)})
    norm = build_part("norm", PartSpec("tanh_norm", "n", {}), width=D)
    w, b = rnd(D, seed=2) * 0.2 + 1.0, rnd(D, seed=3)
    norm.bind({"weight": w.to(DEV), "b": b.to(DEV), "alpha": torch.tensor([0.7], device=DEV)})
    h0, vec = rnd(sum(lens), D, seed=5), rnd(D, seed=6)
    window = torch.zeros((4, taps - 1, D), dtype=torch.float32, device=DEV)
    cache = LayerCache({}, {"c.inputs": window})
    for ones in (False, True):
        ctx = Ctx([1, 1, 1] if ones else lens, [2, 0, 3], dtype)
        rows = 3 if ones else sum(lens)
        stream = ResidualStream(h0[:rows].to(DEV).clone(), ctx, 1, second_buffer=True)
        stream.add_vector(vec.to(DEV))
        window.zero_()
        got = stream.normed_mapped(norm, part, cache)
        x = h0[:rows].double() + vec.double()
        n = (torch.tanh(0.7 * x) * w.double() + b.double()).to(dtype).double()
        want = torch.cat([P.input_conv(p, ker.double()) for p in torch.split(n, [1, 1, 1] if ones else lens)])
        close(got, want, dtype, "map on its own")


def test_stream_keeps_its_meaning_when_its_buffers_change_places():
    """Branches and vectors that wait, a mapped norm (which swaps the buffers), a flush and a plain norm in turn."""
    D, lens, dtype, eps = 64, [7, 5], torch.float32, 1e-3
    part = build_part("input_map", PartSpec("residual_conv", "c", {"taps": 3}), hidden_size=D)
    ker = rnd(D, 3, seed=1, scale=0.6)
    part.bind({"": ker.to(DEV)})
    norm = build_part("norm", PartSpec("rmsnorm", "n", {"eps": eps, "groups": 4, "tensor": ""}), width=D)
    w = rnd(D, seed=2) * 0.2 + 1.0
    norm.bind({"": w.to(DEV)})
    cache = LayerCache({}, {"c.inputs": torch.zeros((2, 2, D), dtype=torch.float32, device=DEV)})
    ctx = Ctx(lens, [0, 1], dtype)
    x = rnd(12, D, seed=5)
    stream = ResidualStream(x.to(DEV).clone(), ctx, 3, second_buffer=True)
    x = x.double()
    for turn in range(3):
        vec, b1, b2, b3 = rnd(D, seed=10 + turn), rnd(12, D, seed=20 + turn), rnd(12, D, seed=30 + turn), rnd(12, D, seed=40 + turn)
        for t, s in ((b1, 0.5), (b2, -1.0), (b3, 2.0)):
            stream.add(t.to(DEV), s)
        stream.add_vector(vec.to(DEV))
        x = x + 0.5 * b1.double() - b2.double() + 2.0 * b3.double() + vec.double()
        n = P.grouped_norm(x, w.double(), eps, 4)
        if turn == 1:
            close(stream.normed(norm), n, dtype, "plain norm")
        else:
            cache.fixed("c.inputs").zero_()
            got = stream.normed_mapped(norm, part, cache)
            close(got, torch.cat([P.input_conv(p, ker.double()) for p in torch.split(n, lens)]), dtype, "mapped norm")
        close(stream.flush(), x, dtype, "stream")


# ----------------------------------------------------------------------------- selective scan
def scan_inputs(T, I, N, R, seed=0):
    x, z = rnd(T, I, seed=seed, scale=1.0), rnd(T, I, seed=seed + 1)
    raw = rnd(T, I, seed=seed + 2)
    B, Cm = rnd(T, N, seed=seed + 3), rnd(T, N, seed=seed + 4)
    a_log = torch.rand(I, N, generator=torch.Generator().manual_seed(seed + 5)) * 6.0 - 5.0   # slow and fast decays
    bias, d = rnd(I, seed=seed + 6) - 1.5, rnd(I, seed=seed + 7)
    return x, z, raw, B, Cm, a_log, bias, d


def plain_scan(x, z, raw, B, Cm, a_log, bias, d, S0):
    """P.selective_scan from a state S0 (put in front as what the zero state has become), gated; also the end state."""
    dt = P.softplus(raw.double() + bias.double())
    A = -torch.exp(a_log.double())
    S, ys = S0.double().clone(), []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t].double())[:, None] * B[t].double()[None, :]
        ys.append(S @ Cm[t].double() + d.double() * x[t].double())
    return torch.stack(ys) * P.silu(z.double()), S


def test_plain_scan_here_is_the_oracles():
    x, z, raw, B, Cm, a_log, bias, d = scan_inputs(17, 6, 3, 2)
    got, _ = plain_scan(x, z, raw, B, Cm, a_log, bias, d, torch.zeros(6, 3))
    want = P.selective_scan(x.double(), P.softplus(raw.double() + bias.double()), -torch.exp(a_log.double()), B.double(), Cm.double(), d.double())
    assert torch.allclose(got, want * P.silu(z.double()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("I,N", [(40, 1), (33, 3), (64, 5), (50, 12), (96, 16), (24, 24), (40, 32), (17, 48), (24, 64), (16, 100), (12, 128), (9, 256)])
def test_selective_scan_walk_from_a_saved_state(dtype, I, N):
    """Portions of one token, of less than a tile and of several tiles in one launch, from states that are not zero, B
    and C anywhere in wider rows, in slots that are not in order."""
    lens, slots = [1, 37, 16, 5], [4, 1, 3, 0]
    T = sum(lens)
    x, z, raw, B, Cm, a_log, bias, d = (t.to(dtype).float() if i < 5 else t for i, t in enumerate(scan_inputs(T, I, N, 4)))
    state0 = rnd(5, I, N, seed=50)
    low = torch.full((T, 2 * N + 11), 3.0)
    off_b, off_c = 8, 8 + N + 3
    low[:, off_b:off_b + N], low[:, off_c:off_c + N] = B, Cm
    wide = torch.cat([x, torch.zeros(T, 3), z], dim=1).to(DEV, dtype)
    ctx = Ctx(lens, slots, dtype)
    state, y = state0.to(DEV).clone(), torch.empty(T, I, dtype=dtype, device=DEV)
    plan = (max(lens), len(lens))
    K.selective_scan(wide[:, :I], raw.to(DEV, dtype), low.to(DEV, dtype), off_b, off_c, wide[:, I + 3:], bias.to(DEV), a_log.to(DEV),
                     d.to(DEV), state, ctx.cu_seqlens, ctx.slots, len(lens), plan, None, y)
    r = 0
    for s, n in enumerate(lens):
        sl = slice(r, r + n)
        want, S = plain_scan(x[sl], z[sl], raw[sl], B[sl], Cm[sl], a_log, bias, d, state0[slots[s]])
        close(y[sl], want, dtype, f"N {N} sequence {s}", bf16=1e-2)
        close(state[slots[s]], S, torch.float32, "state", f32=2e-5)
        r += n
    assert torch.equal(state[2].cpu(), state0[2])


@pytest.mark.parametrize("chunk", [16, 48, 64, 200])
@pytest.mark.parametrize("I,N", [(96, 16), (40, 6), (33, 24), (16, 128)])
def test_selective_scan_in_chunks(chunk, I, N):
    """bfloat16: portions of several chunks, of one and of one token in the same launch; the start states of the chunks
    are passed along the sequence and the end state goes back to the slot."""
    dtype, lens, slots = torch.bfloat16, [333, 1, 64, 65, 15], [2, 0, 1, 4, 3]
    T = sum(lens)
    x, z, raw, B, Cm, a_log, bias, d = (t.to(dtype).float() if i < 5 else t for i, t in enumerate(scan_inputs(T, I, N, 4)))
    a_log -= 2.0                           # slow decays: what a chunk hands to the next matters
    state0 = rnd(5, I, N, seed=50, scale=3.0)
    low = torch.cat([B, Cm], dim=1).to(DEV, dtype)
    ctx = Ctx(lens, slots, dtype)
    state, y = state0.to(DEV).clone(), torch.empty(T, I, dtype=dtype, device=DEV)
    n_chunks = sum(-(-n // chunk) for n in lens)
    scratch = torch.full((n_chunks * I * (N + 1),), 5.0, dtype=torch.float32, device=DEV)
    K.selective_scan(x.to(DEV, dtype), raw.to(DEV, dtype), low, 0, N, z.to(DEV, dtype), bias.to(DEV), a_log.to(DEV), d.to(DEV), state,
                     ctx.cu_seqlens, ctx.slots, len(lens), (chunk, n_chunks), scratch, y)
    r = 0
    for s, n in enumerate(lens):
        sl = slice(r, r + n)
        want, S = plain_scan(x[sl], z[sl], raw[sl], B[sl], Cm[sl], a_log, bias, d, state0[slots[s]])
        close(y[sl], want, dtype, f"chunk {chunk} sequence {s}", bf16=1e-2)
        close(state[slots[s]], S, torch.float32, "state", f32=1e-4)
        r += n


def test_scan_plan_cuts_only_where_the_gpu_would_stay_empty():
    for lens, I, N in (([2048], 512, 16), ([300, 1, 1], 256, 24), ([5000, 4000], 128, 8)):
        chunk, n = K.selective_scan_plan(lens, I, N, torch.bfloat16)
        assert 64 <= chunk < max(lens) and chunk % 16 == 0 and n == sum(-(-k // chunk) for k in lens)
    for lens, I, N, dtype in (([2048], 16384, 16, torch.bfloat16), ([64, 3], 64, 16, torch.bfloat16), ([2048], 512, 16, torch.float32),
                              ([1000] * 16, 2048, 16, torch.bfloat16)):
        assert K.selective_scan_plan(lens, I, N, dtype) == (max(lens), len(lens))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [3, 18])
@pytest.mark.parametrize("I,N,R", [(40, 12, 5), (96, 16, 8), (33, 1, 3), (64, 40, 24), (24, 128, 64), (10, 256, 1)])
def test_selective_step_makes_its_step_sizes(dtype, I, N, R, n):
    slots = [(5 * s + 2) % (n + 1) for s in range(n)] if n == 18 else [2, 0, 3]
    x, z, _, B, Cm, a_log, bias, d = (t.to(dtype).float() if i < 5 else t for i, t in enumerate(scan_inputs(n, I, N, R)))
    t_low, w_dt = rnd(n, R, seed=60), rnd(I, R, seed=61, scale=R ** -0.5)
    off_b, off_c = (R + 7) // 8 * 8, (R + 7) // 8 * 8 + (N + 7) // 8 * 8
    low = torch.zeros(n, off_c + (N + 7) // 8 * 8)
    low[:, :R], low[:, off_b:off_b + N], low[:, off_c:off_c + N] = t_low, B, Cm
    state0 = rnd(n + 1, I, N, seed=50)
    state, y = state0.to(DEV).clone(), torch.empty(n, I, dtype=dtype, device=DEV)
    K.selective_step(x.to(DEV, dtype), low.to(DEV, dtype), R, off_b, off_c, w_dt.to(DEV, dtype), z.to(DEV, dtype), bias.to(DEV),
                     a_log.to(DEV), d.to(DEV), state, i32(slots), y)
    raw = t_low.double() @ w_dt.double().t()
    given = raw.to(dtype)      # the same with the step sizes made before
    state2, y2 = state0.to(DEV).clone(), torch.empty(n, I, dtype=dtype, device=DEV)
    K.selective_step(x.to(DEV, dtype), low.to(DEV, dtype), R, off_b, off_c, w_dt.to(DEV, dtype), z.to(DEV, dtype), bias.to(DEV),
                     a_log.to(DEV), d.to(DEV), state2, i32(slots), y2, raw=given.to(DEV))
    for s in range(n):
        want, S = plain_scan(x[s:s + 1], z[s:s + 1], given.double()[s:s + 1], B[s:s + 1], Cm[s:s + 1], a_log, bias, d, state0[slots[s]])
        close(y2[s:s + 1], want, dtype, "step, sizes given", bf16=1e-2)
        close(state2[slots[s]], S, torch.float32, "state, sizes given")
    for s in range(n):
        want, S = plain_scan(x[s:s + 1], z[s:s + 1], raw[s:s + 1], B[s:s + 1], Cm[s:s + 1], a_log, bias, d, state0[slots[s]])
        close(y[s:s + 1], want, dtype, "step", bf16=1e-2)
        close(state[slots[s]], S, torch.float32, "state")
    left = (set(range(n + 1)) - set(slots)).pop()
    assert torch.equal(state[left].cpu(), state0[left])


# ----------------------------------------------------------------------------- attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,rot_dims,norm_v", [(4, 2, 24, 16, 16, True), (3, 3, 8, 40, 8, True), (6, 1, 64, 64, 64, True),
                                                      (4, 4, 20, 12, 0, True), (4, 2, 24, 16, 16, False)])
def test_scaled_rotation_and_normed_values_into_the_pages(dtype, H, G, d, dv, rot_dims, norm_v):
    """Positions up to 5,000 in two sequences whose pages are not in order: the queries, and what the pages hold
    afterwards (turned keys; value rows over their own root mean square, head by head)."""
    page, eps = 16, 1e-2
    Dp = (max(d, dv) + 15) // 16 * 16
    positions = [0, 1, 15, 16, 17, 999, 5000, 5, 31, 32]
    seq = [0] * 7 + [1] * 3
    T = len(positions)
    scaling = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}
    from poor_mans_mamba_b200.parts.rope import rotary_frequencies
    inv = rotary_frequencies(rot_dims, 1000.0, scaling=tuple(scaling.values())).to(DEV) if rot_dims else None
    wide = rnd(T, (H + G) * d + G * dv + 5, seed=1, scale=2.0)
    wide[:, (H + G) * d:(H + G) * d + dv] *= 10.0     # the first value head is much larger than the others
    wide = wide.to(DEV, dtype)
    q, k, v = wide[:, :H * d], wide[:, H * d:(H + G) * d], wide[:, (H + G) * d:(H + G) * d + G * dv]
    n_blocks = 5000 // page + 1
    table = torch.randperm(2 * n_blocks, generator=torch.Generator().manual_seed(7)).to(torch.int32).view(2, n_blocks).to(DEV)
    pool = torch.full((2 * n_blocks, 2, page, G * Dp), 7.0, dtype=dtype, device=DEV)  # pages used before
    q_out = torch.full((T, H * Dp), 5.0, dtype=dtype, device=DEV)
    K.rope_pairs_store(q, k, v, inv, rot_dims, i32(positions), i32(seq), table, pool, q_out, H, G, d, dv, Dp, half_layout=True,
                       v_norm_eps=eps if norm_v else None)
    pos = torch.tensor(positions)
    freq = P.frequencies(rot_dims, 1000.0, scaling).float().double()   # the stored frequencies: at 5,000 their rounding shows
    want_q = P.rotate_halves(q.double().cpu().view(T, H, d), pos, freq)
    want_k = P.rotate_halves(k.double().cpu().view(T, G, d), pos, freq)
    want_v = v.double().cpu().view(T, G, dv)
    want_v = P.rms(want_v, eps) if norm_v else want_v
    close(q_out.view(T, H, Dp)[:, :, :d], want_q, dtype, "queries", f32=3e-4)
    for t in range(T):
        pg = int(table[seq[t], positions[t] // page])
        row_k, row_v = (pool[pg, plane, positions[t] % page].view(G, Dp) for plane in (0, 1))
        close(row_k[:, :d], want_k[t], dtype, "key row", f32=3e-4)
        close(row_v[:, :dv], want_v[t], dtype, "value row")
        assert float(row_k[:, d:].abs().sum()) == 0.0 and float(row_v[:, dv:].abs().sum()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [0, 1, 7, 33])
def test_window_with_a_sink_at_its_edges(dtype, window):
    """The attention part over 90 tokens in portions: the last key inside every window and the first outside it are
    loud, and the sinks lie at the level of the loud scores."""
    D, T = 40, 90
    m = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 12, "scale": 0.3, "rot": {"dims": 8, "base": 100.0, "scaling": {
        "factor": 4.0, "low": 1.0, "high": 4.0, "original": 40}}, "mask": {"size": window}}
    W = {"q": rnd(64, D, seed=1, scale=0.3), "k": rnd(32, D, seed=2, scale=0.3), "v": rnd(24, D, seed=3, scale=0.3),
         "sink": rnd(4, seed=4) + 3.0, "o": rnd(D, 48, seed=5, scale=0.2)}
    W["q"][15] *= 4.0       # the first head's last unturned entry carries single scores far above the rest
    W["k"][15] *= 4.0
    part = build_part("mixer", PartSpec("rotary_gated_attention", "mix", {
        "heads": 4, "kv_heads": 2, "dim": 16, "vdim": 12, "rot_dims": 8, "rot_base": 100.0, "rot_scaling": (4.0, 1.0, 4.0, 40),
        "scale": 0.3, "bias": False, "gate": False, "window": window, "sink": True, "value_norm_eps": 1e-3}), hidden_size=D)
    part.bind({k: w.to(DEV, torch.float32 if k == "sink" else dtype) for k, w in W.items()})
    part.finalize(dtype, torch.device(DEV))
    x = rnd(T, D, seed=9)
    W64 = {k: v.double() for k, v in W.items()}
    want = P.attention(x.double(), W64, "", m, 1e-3, torch.arange(T))
    for other in (dict(m, mask={"size": window + 1}), dict(m, mask={"size": window - 1})):
        if window > 1:
            assert float((P.attention(x.double(), W64, "", other, 1e-3, torch.arange(T)) - want).abs().max()) > 0.1
    quiet = dict(W64, sink=W64["sink"] - 50.0)
    assert float((P.attention(x.double(), quiet, "", m, 1e-3, torch.arange(T)) - want).abs().max()) > 0.1
    from poor_mans_mamba_b200.cache import CacheManager
    from poor_mans_mamba_b200.engine.context import StepContext
    cache = CacheManager({0: [(f"mix.{s.name}", s) for s in part.state_specs()]}, 16, 8, 1, dtype, DEV)
    cache.admit("r")
    at = 0
    for n in (1, 30, 2, 1, 1, 40, 15):
        cache.grow("r", at + n)
        tables = {k: i32([[p if p >= 0 else g.num_pages for p in g.tables["r"]]]) for k, g in cache.groups.items()}
        ws = Workspace(torch.device(DEV))
        ctx = StepContext(n_tokens=n, n_seq=1, tokens=i32([0] * n), positions=i32(list(range(at, at + n))), seq_of=i32([0] * n),
                          cu_seqlens=i32([0, n]), slots=i32([0]), logit_rows=i32([]), n_rows=0, decode_only=n == 1,
                          kv_len_bound=at + n, dtype=dtype, workspace=ws, new_lens=[n], past_lens=[at])
        out = torch.empty(n, D, dtype=dtype, device=DEV)
        part.forward(x[at:at + n].to(DEV, dtype), ctx, cache.layer_caches(tables)[0], out)
        close(out, want[at:at + n], dtype, f"window {window} tokens {at}..{at + n}", f32=3e-5, bf16=3e-2)
        at += n
        cache.advance("r", n)
    assert at == T


# ----------------------------------------------------------------------------- routed feed-forward
@pytest.mark.parametrize("E,top", [(8, 1), (6, 2), (12, 5), (4, 4), (64, 6)])
@pytest.mark.parametrize("T", [7, 700])
def test_router_keeps_its_sigmoid_scores(E, top, T):
    D = 40
    x, w = rnd(T, D, seed=E + T), rnd(E, D, seed=top, scale=0.3)
    ids = torch.empty(T, top, dtype=torch.int32, device=DEV)
    weights = torch.empty(T, top, dtype=torch.float32, device=DEV)
    K.moe_route(x.to(DEV), w.to(DEV), None, top, ids, weights, scored="sigmoid")
    z = x.double() @ w.double().t()
    checked = 0
    for t in range(T):
        order = z[t].sort().values
        if float((order[1:] - order[:-1]).min()) < 1e-4:
            continue  # a close call: either choice is right
        chosen, ws = P.route(z[t], top)
        assert ids[t].tolist() == chosen, f"token {t}"
        close(weights[t], torch.stack(ws), torch.float32, "weights", f32=1e-5)
        checked += 1
    assert checked > T // 3


@pytest.mark.parametrize("form,T,D,F", [("float", 9, 36, 20), ("float", 40, 64, 24), ("mma_few", 12, 64, 40), ("mma", 300, 64, 72), ("tcgen05", 300, 128, 64)])
def test_score_weights_the_experts_input(form, T, D, F):
    """The weight enters before the activation (silu(w g) * (w u) is no multiple of silu(g) * u), in every form of the
    grouped product, float32 for the float form and bfloat16 for the others."""
    E, top = 5, 2
    dtype = torch.float32 if form == "float" else torch.bfloat16
    x = rnd(T, D, seed=1)
    gate_up = rnd(E, 2 * F, D, seed=2, scale=2.0 * D ** -0.5)
    g = torch.Generator().manual_seed(3)
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    ids[ids == 3] = 1                       # an expert without tokens
    wts = torch.rand(T, top, generator=g) * 0.9 + 0.05
    A = T * top
    offsets, tile_start, perm = (torch.empty(n, dtype=torch.int32, device=DEV) for n in (E + 1, E + 1, A))
    K.moe_plan(ids.to(DEV), E, form, offsets, tile_start, perm)
    act = torch.empty(A, F, dtype=dtype, device=DEV)
    xd, wd, rw = x.to(DEV, dtype), gate_up.to(DEV, dtype), wts.to(DEV)
    if form == "tcgen05":
        xs = torch.empty(A, D, dtype=dtype, device=DEV)
        K.moe_gather_rows(xd, perm, top, xs)
        K.moe_tc_gemm(xs, wd, perm, offsets, tile_start, True, act, limit=math.inf, alpha=1.0, shift=0.0, row_weights=rw)
        torch.cuda.synchronize()
        assert K.tc_gemm_status(xd.device) == 0
    else:
        K.moe_gemm(xd, wd, perm, offsets, tile_start, top, True, act, form, limit=math.inf, alpha=1.0, shift=0.0, row_weights=rw)
    got = act.double().cpu()
    for i, p in enumerate(perm.tolist()):
        t, j = divmod(p, top)
        e = int(ids[t, j])
        h = float(wts[t, j]) * (gate_up[e].double() @ x[t].double())
        close(got[i], P.silu(h[:F]) * h[F:], dtype, f"pair {p}", bf16=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,D,F,shared", [(5, 48, 20, 24), (5, 48, 20, 0), (90, 64, 64, 32), (600, 128, 64, 128)])
def test_routed_feed_forward_with_a_shared_expert(dtype, T, D, F, shared):
    E, top = 6, 2
    part = build_part("feed_forward", PartSpec("routed_glu", "mlp", {
        "experts": E, "top": top, "expert_ff": F, "expert_limit": math.inf, "shared_ff": shared, "shared_limit": math.inf,
        "act_alpha": 1.0, "act_shift": 0.0, "router_bias": False, "router": "sigmoid", "weigh": "input"}), hidden_size=D)
    W = {}
    for i, spec in enumerate(part.param_specs()):
        W[spec.name] = rnd(*spec.shape, seed=i, scale=1.5 * spec.shape[-1] ** -0.5)
    x = rnd(T, D, seed=77)
    x[:, 0] = x[:, 0].abs() + 2.0
    W["router"] *= 0.1
    W["router"][:, 0] = torch.tensor([0.3, -0.6, 0.9, -0.3, 0.0, 0.6]).to(torch.bfloat16).float()   # no close call
    part.bind({k: v.to(DEV, torch.float32 if k == "router" else dtype) for k, v in W.items()})
    part.finalize(dtype, torch.device(DEV))
    ctx = Ctx([T], [0], dtype)
    out = torch.empty(T, D, dtype=dtype, device=DEV)
    part.forward(x.to(DEV, dtype), ctx, out)
    mlp = {"router": {"top": top}, "shared": {"ff": shared} if shared else None}
    want = P.routed_ffn(x.double(), {k: v.double() for k, v in W.items()}, "", mlp)
    close(out, want, dtype, "routed feed-forward", bf16=2e-2)


# ----------------------------------------------------------------------------- output
@pytest.mark.parametrize("cap,scale", [(3.0, 1.0), (30.0, 0.5)])
def test_softcap_of_the_logits(cap, scale):
    x, w = rnd(5, 64, seed=1), rnd(77, 64, seed=2)
    want = cap * torch.tanh(scale * (x.double() @ w.double().t()) / cap)
    out = torch.empty(5, 77, dtype=torch.float32, device=DEV)
    K.skinny_linear_f32(x.to(DEV, torch.bfloat16), w.to(DEV, torch.bfloat16), out, scale, cap)
    close(out, want, torch.float32, "in the epilogue of the head", f32=1e-5)
    out = (x @ w.t()).to(DEV).contiguous()
    K.softcap_f32_(out, scale, cap)
    close(out, want, torch.float32, "on its own", f32=1e-5)
    K.skinny_linear_f32(x.to(DEV, torch.bfloat16), w.to(DEV, torch.bfloat16), out, scale)
    close(out, scale * (x.double() @ w.double().t()), torch.float32, "no cap", f32=1e-5)
