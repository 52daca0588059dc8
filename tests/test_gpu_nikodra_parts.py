"""Each mechanism of the Nikodra parts alone against its plain function (GPU): the kernels are called as the model
calls them, on inputs made so that a fault shows."""
import math

import pytest
import torch

from plain import nikodra_plain as P

from poor_mans_mamba_b200.cache import CacheManager
from poor_mans_mamba_b200.engine.context import StepContext
from poor_mans_mamba_b200.engine.workspace import Workspace
from poor_mans_mamba_b200.kernels import ops as K
from poor_mans_mamba_b200.parts.base import LayerCache, PartSpec, build_part
from poor_mans_mamba_b200.parts.block import ResidualStream
from poor_mans_mamba_b200.parts.rope import rotary_frequencies, yarn_frequencies
import poor_mans_mamba_b200.parts  # noqa: F401  (registration)

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
F64 = torch.float64


def rnd(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(torch.bfloat16).float()


def close(got, want, dtype, what, f32=2e-5, bf16=2e-2):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} vs {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: not finite"
    tol = (f32 if dtype == torch.float32 else bf16) * max(1.0, float(want.abs().max()))
    err = float((got - want).abs().max())
    assert err <= tol, f"{what}: {err:.3e} > {tol:.3e}"


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


class Steps:
    """Walks requests of given lengths through steps whose portions are given, with a context as the engine makes it:
    ``cuts[s]`` lists the tokens request s brings to each step (0: it sits out)."""

    def __init__(self, cuts, slots, dtype, past=None):
        self.cuts, self.slots, self.dtype = cuts, slots, dtype
        self.at = list(past) if past else [0] * len(cuts)

    def __iter__(self):
        for step in range(len(self.cuts[0])):
            live = [s for s in range(len(self.cuts)) if self.cuts[s][step] > 0]
            lens = [self.cuts[s][step] for s in live]
            cu = [0]
            for n in lens:
                cu.append(cu[-1] + n)
            ctx = StepContext(
                n_tokens=cu[-1], n_seq=len(live), tokens=i32([0] * cu[-1]),
                positions=i32([self.at[s] + j for s, n in zip(live, lens) for j in range(n)]),
                seq_of=i32([q for q, n in enumerate(lens) for _ in range(n)]), cu_seqlens=i32(cu),
                slots=i32([self.slots[s] for s in live]), logit_rows=i32([]), n_rows=0, decode_only=all(n == 1 for n in lens),
                kv_len_bound=max(self.at[s] + n for s, n in zip(live, lens)), dtype=self.dtype,
                workspace=Workspace(torch.device(DEV)), new_lens=lens, past_lens=[self.at[s] for s in live])
            yield ctx, [(s, self.at[s], n) for s, n in zip(live, lens)]
            for s, n in zip(live, lens):
                self.at[s] += n


CUTS = [[1, 2, 40, 1, 90, 8], [5, 1, 1, 39, 1, 0], [0, 20, 1, 1, 1, 0], [0, 1, 0, 64, 33, 0]]
LENGTHS = [sum(c) for c in CUTS]
SLOTS = [3, 0, 2, 5]


# ----------------------------------------------------------------------------- embedding
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,buckets,mul_prev,mul_cur,V", [(50, 7, 3, 2, 40), (96, 1009, 100003, 77, 30000), (8, 1, 5, 0, 9)])
def test_bigram_rows_follow_the_token_before_in_any_cut(dtype, D, buckets, mul_prev, mul_cur, V):
    """Every cut, slots used before, products of ids and multipliers beyond 32 bits."""
    g = torch.Generator().manual_seed(3)
    seqs = [torch.randint(0, V, (n,), generator=g).tolist() for n in LENGTHS]
    table, extra = rnd(V, D, seed=1), rnd(buckets + 1, D, seed=2)
    w = rnd(D, seed=5) * 0.2 + 1.0
    W = {"embed": table.double(), "bigram": extra.double()}
    want = [P.embed(s, W, {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}) for s in seqs]
    previous = torch.full((7, 1), 77, dtype=torch.int32, device=DEV)
    for normed in (False, True):
        previous[SLOTS] = 0
        for ctx, live in Steps(CUTS, SLOTS, dtype):
            toks = i32([t for s, a, n in live for t in seqs[s][a:a + n]])
            out = torch.full((ctx.n_tokens, D), 9.0, device=DEV)
            K.embed(out, table.to(DEV, dtype), toks, 1.0, w.to(DEV) if normed else None, 1e-3,
                    bigram=(extra.to(DEV, dtype), mul_prev, mul_cur), previous=previous, seq_of=ctx.seq_of, cu=ctx.cu_seqlens, slots=ctx.slots)
            ref = torch.cat([want[s][a:a + n] for s, a, n in live])
            close(out, P.rms(ref, 1e-3) * w.double() if normed else ref, torch.float32, "embedding", f32=3e-6)
            for s, a, n in live:
                assert int(previous[SLOTS[s], 0]) == seqs[s][a + n - 1] + 1
    assert int(previous[1, 0]) == 77


# ----------------------------------------------------------------------------- norms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [50, 72, 1024, 3072, 6000])
def test_post_norm_with_a_bias_and_a_multiplier(dtype, D):
    """x + m norm_b(branch + bias), then the next norm: one launch; the bias alone is as large as the branch."""
    T, eps, m = 7, 1e-3, 0.4
    x0, branch, bias = rnd(T, D, seed=1, scale=2.0), rnd(T, D, seed=2).to(dtype).float(), rnd(D, seed=3, scale=2.0)
    wb, wn = rnd(D, seed=4, scale=0.3), rnd(D, seed=5, scale=0.3)
    post = build_part("norm", PartSpec("rmsnorm", "b", {"eps": eps, "offset": 1.0, "tensor": "", "multiplier": m}), width=D)
    nxt = build_part("norm", PartSpec("rmsnorm", "n", {"eps": eps, "offset": 1.0, "tensor": ""}), width=D)
    post.bind({"": wb.to(DEV)})
    nxt.bind({"": wn.to(DEV)})
    x = x0.double() + m * P.norm(branch.double() + bias.double(), wb.double(), eps)
    for way in ("normed", "rows", "flush", "settled", "plain"):
        ctx = StepContext(*([None] * 8), n_rows=0, decode_only=False, kv_len_bound=1, dtype=dtype, workspace=Workspace(torch.device(DEV)))
        stream = ResidualStream(x0.to(DEV).clone(), ctx, 3)
        stream.add_normed([(branch.to(DEV, dtype), 1.0)], post, None if way == "plain" else bias.to(DEV))
        if way == "normed":
            close(stream.normed(nxt), P.norm(x, wn.double(), eps), dtype, way, bf16=1e-2)
            close(stream.flush(), x, torch.float32, "stream")
        elif way == "rows":
            close(stream.normed(nxt, rows=i32([5, 0])), P.norm(x, wn.double(), eps)[[5, 0]], dtype, way, bf16=1e-2)
            close(stream.flush(), x, torch.float32, "stream after chosen rows")
        elif way == "flush":
            close(stream.flush(), x, torch.float32, way)
        elif way == "settled":   # another branch arrives before any norm
            other = rnd(T, D, seed=9).to(dtype).float()
            stream.add(other.to(DEV, dtype), 0.5)
            close(stream.flush(), x + 0.5 * other.double(), dtype, way, bf16=1e-2)
        else:
            close(stream.flush(), x0.double() + m * P.norm(branch.double(), wb.double(), eps), torch.float32, way)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("groups,width,gate", [(3, 16, "silu"), (5, 12, "sigmoid"), (2, 200, "silu"), (4, 256, "silu"), (2, 300, "sigmoid"), (1, 64, "silu")])
def test_norm_of_every_head_then_the_gate(dtype, groups, width, gate):
    T, I, eps = 19, groups * width, 1e-2
    y, z, w = rnd(T, I, seed=1, scale=2.0), rnd(T, I + 3, seed=2, scale=2.0).to(dtype).float(), rnd(I, seed=3) * 0.3 + 1.0
    y[:, :width] *= 30.0      # one head much larger than the others
    out = torch.empty(T, I, dtype=dtype, device=DEV)
    K.gated_norm(y.to(DEV), z.to(DEV, dtype)[:, 3:], 1.0, None, w.to(DEV), eps, groups, True, out, gate=gate)
    zz = z[:, 3:].double()
    g = P.silu(zz) if gate == "silu" else torch.sigmoid(zz)
    close(out, P.rms(y.double().view(T, groups, width), eps).reshape(T, I) * w.double() * g, dtype, "gated norm", bf16=1e-2)


# ----------------------------------------------------------------------------- attention: preparation
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,rot,halves,norm,bias,mix", [
    (6, 2, 24, 16, 16, False, "weight", True, "later"), (3, 3, 8, 40, 8, False, "weight", True, "first"), (8, 1, 64, 64, 64, False, "weight", True, "later"),
    (4, 4, 20, 12, 0, False, "unit", False, None), (2, 1, 128, 96, 32, True, "unit", True, None), (2, 2, 250, 256, 250, False, "weight", False, "later"),
    (5, 1, 16, 16, 6, True, None, True, "first")])
def test_head_norms_rotation_and_mixed_values_into_the_pages(dtype, H, G, d, dv, rot, halves, norm, bias, mix):
    page, eps, yarn = 16, 1e-2, (8.0, 64.0, 4.0, 0.5)
    Dp = (max(d, dv) + 15) // 16 * 16
    positions, seq = [0, 1, 15, 16, 17, 999, 5000, 5, 31, 32], [0] * 7 + [1] * 3
    T = len(positions)
    inv, amp = yarn_frequencies(rot, 1000.0, *yarn) if rot else (None, 1.0)
    wide = rnd(T, (H + G) * d + G * dv + 5, seed=1, scale=2.0)
    wide[:, :d] *= 10.0     # the first query head is much larger than the others
    wide = wide.to(DEV, dtype)
    q, k, v = wide[:, :H * d], wide[:, H * d:(H + G) * d], wide[:, (H + G) * d:(H + G) * d + G * dv]
    biases = tuple(rnd(n, seed=20 + i, scale=2.0).to(DEV) for i, n in enumerate((H * d, G * d, G * dv))) if bias else None
    weights = (torch.rand(d) * 1.5 + 0.5, torch.rand(d) * 1.5 + 0.5) if norm == "weight" else None
    lam = torch.tensor([0.3])
    v0 = rnd(T, G * dv, seed=30, scale=3.0).to(dtype)
    values = None if mix is None else (v0 if mix == "later" else torch.full_like(v0, 9.0)).to(DEV)
    n_blocks = 5000 // page + 1
    table = torch.randperm(2 * n_blocks, generator=torch.Generator().manual_seed(7)).to(torch.int32).view(2, n_blocks).to(DEV)
    pool = torch.full((2 * n_blocks, 2, page, G * Dp), 7.0, dtype=dtype, device=DEV)  # pages used before
    q_out = torch.full((T, H * Dp), 5.0, dtype=dtype, device=DEV)
    K.head_norm_rope_store(q, k, v, inv.to(DEV) if rot else None, rot, i32(positions), i32(seq), table, pool, q_out, H, G, d, dv, Dp,
                           half_layout=halves, amplitude=amp, biases=biases, norm_eps=None if norm is None else eps,
                           norm_weights=None if weights is None else tuple(w.to(DEV) for w in weights), values=values,
                           mix_weight=lam.to(DEV) if mix == "later" else None)
    pos = torch.tensor(positions)
    freq = inv.double() if rot else torch.zeros(0, dtype=F64)   # the stored frequencies: at 5,000 their rounding shows

    def prepared(x, n, i):
        x = x.double().cpu().view(T, n, d)
        if bias:
            x = x + biases[i].double().cpu().view(n, d)
        if norm is not None:
            x = P.rms(x, eps) * (weights[i].double() if weights else 1.0)
        return P.rotate(x, pos, freq, halves, amp)
    want_v = v.double().cpu().view(T, G, dv)
    if bias:
        want_v = want_v + biases[2].double().cpu().view(G, dv)
    if mix == "first":
        close(values.view(T, G, dv), want_v, dtype, "values left for later layers")
    if mix == "later":
        want_v = 0.7 * want_v + 0.3 * v0.double().view(T, G, dv)
        assert torch.equal(values.cpu(), v0)
    close(q_out.view(T, H, Dp)[:, :, :d], prepared(q, H, 0), dtype, "queries", f32=3e-4)
    assert float(q_out.view(T, H, Dp)[:, :, d:].abs().sum()) == 0.0
    want_k = prepared(k, G, 1)
    for t in range(T):
        pg = int(table[seq[t], positions[t] // page])
        row_k, row_v = (pool[pg, plane, positions[t] % page].view(G, Dp) for plane in (0, 1))
        close(row_k[:, :d], want_k[t], dtype, "key row", f32=3e-4)
        close(row_v[:, :dv], want_v[t], dtype, "value row")
        assert float(row_k[:, d:].abs().sum()) == 0.0 and float(row_v[:, dv:].abs().sum()) == 0.0


# ----------------------------------------------------------------------------- attention: chunks and the one more
def run_part(part, x, cuts, slots, dtype, page_size, num_pages, n_slots=6, carried=None):
    """The mixer over the requests' rows x[s] in every step; the outputs per request."""
    D = x[0].shape[1]
    cache = CacheManager({0: [(f"mix.{s.name}", s) for s in part.state_specs()]}, page_size, num_pages, n_slots, dtype, DEV)
    outs = [torch.full((t.shape[0], D), float("nan"), dtype=F64) for t in x]
    done = [0] * len(x)
    seen = set()
    steps = Steps(cuts, slots, dtype)
    for ctx, live in steps:
        for s, a, n in live:
            if s not in seen:
                seen.add(s)
                cache.admit(s)
            cache.grow(s, a + n)
        ctx.slots = i32([cache.slot(s) for s, _, _ in live])
        tables = {k: i32([[(p if p >= 0 else g.num_pages) for p in g.tables[s]] + [g.num_pages] * (max(len(g.tables[q]) for q, _, _ in live) - len(g.tables[s]))
                          for s, _, _ in live]) for k, g in cache.groups.items()}
        if carried is not None:
            ctx.carried = {k: torch.cat([v[s][a:a + n] for s, a, n in live]).to(DEV, dtype) for k, v in carried.items()}
        rows = torch.cat([x[s][a:a + n] for s, a, n in live]).to(DEV, dtype)
        out = torch.empty(ctx.n_tokens, D, dtype=dtype, device=DEV)
        part.forward(rows, ctx, cache.layer_caches(tables)[0], out)
        K.check_status(torch.device(DEV), wait=True)
        r = 0
        for s, a, n in live:
            outs[s][a:a + n] = out[r:r + n].double().cpu()
            r += n
            done[s] += n
            cache.advance(s, n)
            if done[s] == x[s].shape[0]:
                cache.release(s)
        cache.check()
    return outs


def loud_left(D, H, G, d, dv):
    """Projections under which keys stand out far: one entry of every head follows one input channel, which is large at
    some tokens only."""
    W = {"q": rnd(H * d, D, seed=1, scale=0.3), "k": rnd(G * d, D, seed=2, scale=0.3), "v": rnd(G * dv, D, seed=3, scale=0.3),
         "o": rnd(D, H * dv, seed=5, scale=0.3)}
    return W


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,chunk", [(4, 2, 16, 24, 1), (4, 2, 16, 24, 7), (6, 1, 48, 16, 16), (4, 1, 64, 64, 33), (3, 3, 8, 8, 0), (8, 2, 128, 96, 40)])
def test_chunked_attention_at_its_edges(dtype, H, G, d, dv, chunk):
    """Unit-norm queries and keys with a scale at which single keys take nearly all the weight, over portions that cut
    the chunks and pages anywhere; a chunk one token longer or shorter, or no one in the denominator, would show."""
    D = 40
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": 6.0 / d, "mask": {"size": chunk}}
    W = loud_left(D, H, G, d, dv)
    part = build_part("mixer", PartSpec("head_norm_attention", "mix", {
        "heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": m["scale"], "norm_eps": 1e-3, "qk_norm": "unit", "chunk": chunk,
        "one_more": True}), hidden_size=D)
    part.bind({k: w.to(DEV, dtype) for k, w in W.items()})
    part.finalize(dtype, torch.device(DEV))
    x = [rnd(n, D, seed=40 + i, scale=1.5) for i, n in enumerate(LENGTHS)]
    W64 = {k: v.double() for k, v in W.items()}
    want = [P.chunked_attention(t.double(), W64, "", m, 1e-3) for t in x]
    for other in (chunk + 1, chunk - 1):
        if chunk > 1:
            moved = P.chunked_attention(x[0].double(), W64, "", dict(m, mask={"size": other}), 1e-3)
            assert float((moved - want[0]).abs().max()) > 0.1
    for page in (16, 64):
        got = run_part(part, x, CUTS, SLOTS, dtype, page, 24)
        for s, ref in enumerate(want):
            close(got[s], ref, dtype, f"chunk {chunk} page {page} sequence {s}", f32=3e-5, bf16=3e-2)


@pytest.mark.parametrize("H,G,d,chunk", [(8, 2, 64, 100), (8, 2, 64, 64), (4, 1, 128, 200), (4, 2, 64, 700), (16, 1, 64, 37)])
def test_chunks_on_the_tensor_core_kernels(H, G, d, chunk):
    """Prompt portions of hundreds of tokens (the tcgen05 form), short ones and single tokens at positions on both sides
    of chunk edges, against the plain attention."""
    D, dtype = 64, torch.bfloat16
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": 5.0 / d, "mask": {"size": chunk}}
    W = loud_left(D, H, G, d, d)
    part = build_part("mixer", PartSpec("head_norm_attention", "mix", {
        "heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": m["scale"], "norm_eps": 1e-3, "qk_norm": "unit", "chunk": chunk,
        "one_more": True}), hidden_size=D)
    part.bind({k: w.to(DEV, dtype) for k, w in W.items()})
    part.finalize(dtype, torch.device(DEV))
    assert K.attention_tc_supported(H, G, d, 64)
    cuts = [[300, 1, 1, 98, 301, 1, 1, 1], [0, 260, 1, 2, 37, 1, 1, 1]]
    x = [rnd(sum(c), D, seed=70 + i, scale=1.5) for i, c in enumerate(cuts)]
    W64 = {k: v.double() for k, v in W.items()}
    got = run_part(part, x, cuts, [0, 1], dtype, 64, 24)
    for s, t in enumerate(x):
        close(got[s], P.chunked_attention(t.double(), W64, "", m, 1e-3), dtype, f"sequence {s}", bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mix", [None, "first", "later"])
def test_attention_with_norms_scaled_rotation_and_mixed_values(dtype, mix):
    """The whole mixer: one key of every request is turned to score far above the rest wherever it lies; biases,
    amplitude, mixing and the one in the denominator all show when left out of the oracle."""
    D, H, G, d, dv, eps = 40, 6, 2, 24, 16, 1e-3
    yarn = (8.0, 40.0, 4.0, 0.5)
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": 0.35, "v_mix": mix is not None,
         "rot": {"dims": 16, "base": 300.0, "scaling": dict(zip(("factor", "original", "fast", "slow"), yarn))}}
    W = {"q": rnd(H * d, D, seed=1, scale=0.3), "k": rnd(G * d, D, seed=2, scale=0.3), "v": rnd(G * dv, D, seed=3, scale=0.3),
         "o": rnd(D, H * dv, seed=5, scale=0.3), "q.b": rnd(H * d, seed=6, scale=0.7), "k.b": rnd(G * d, seed=7, scale=0.7),
         "v.b": rnd(G * dv, seed=8, scale=0.7), "o.b": rnd(D, seed=9), "q.norm": torch.rand(d) + 0.5, "k.norm": torch.rand(d) + 0.5,
         "vmix": torch.tensor(0.6)}
    W["q.norm"][-1] = W["k.norm"][-1] = 3.0      # an unturned entry that decides scores
    W["q.norm"][14] = W["k.norm"][14] = 2.0      # and a slowly turning one
    names = {"value_mix": mix, "carried_values": "v0"} if mix else {}
    part = build_part("mixer", PartSpec("head_norm_attention", "mix", {
        "heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": m["scale"], "norm_eps": eps, "bias": True, "qk_norm": "weight",
        "rot_dims": 16, "rot_base": 300.0, "rot_yarn": yarn, "one_more": True, **names}), hidden_size=D)
    part.bind({ps.name: W[ps.name].to(DEV, dtype if ps.kind == "matrix" else torch.float32) for ps in part.param_specs()})
    part.finalize(dtype, torch.device(DEV))
    x = [rnd(n, D, seed=40 + i, scale=1.2) for i, n in enumerate(LENGTHS)]
    v0 = [rnd(n, G * dv, seed=60 + i) for i, n in enumerate(LENGTHS)]
    W64 = {k: v.double() for k, v in W.items()}

    def plain(s, weights=W64, cfg=m):
        shared = {"v": v0[s].double().view(-1, G, dv)} if mix == "later" else {}
        return P.attention(x[s].double(), weights, "", cfg, eps, torch.arange(LENGTHS[s]), shared)
    want = [plain(s) for s in range(len(x))]
    for change in ({"q.b": W64["q.b"] * 0}, {"v.b": W64["v.b"] * 0}, {"o.b": W64["o.b"] * 0}) + (({"vmix": W64["vmix"] * 0},) if mix == "later" else ()):
        assert float((plain(0, dict(W64, **change)) - want[0]).abs().max()) > 0.15
    unscaled = dict(m, rot={"dims": 16, "base": 300.0})
    assert float((plain(0, cfg=unscaled) - want[0]).abs().max()) > 0.15
    carried = None
    if mix is not None:
        carried = {"v0": v0}
    got = run_part(part, x, CUTS, SLOTS, dtype, 16, 24, carried=carried)
    for s, ref in enumerate(want):
        close(got[s], ref, dtype, f"mix {mix} sequence {s}", f32=4e-5, bf16=3e-2)


# ----------------------------------------------------------------------------- recurrences
def walk_retention(q, k, v, decay, S):
    o = []
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        o.append(q[t] @ S)
    return torch.stack(o), S


def walk_wkv(r, k, v, w, u, S):
    o = []
    for t in range(r.shape[0]):
        kv = torch.outer(k[t], v[t])
        o.append(r[t] @ (S + u[:, None] * kv))
        S = w[t][:, None] * S + kv
    return torch.stack(o), S


def test_plain_walks_here_are_the_oracles():
    q, k, v, w = (rnd(13, 1, n, seed=i).double() for i, n in enumerate((6, 6, 4, 6)))
    u = rnd(1, 6, seed=9).double()
    assert torch.allclose(walk_retention(q[:, 0], k[:, 0], v[:, 0], 0.7, torch.zeros(6, 4, dtype=F64))[0], P.retention_scan(q, k, v, [0.7])[:, 0])
    w = torch.sigmoid(w)
    assert torch.allclose(walk_wkv(q[:, 0], k[:, 0], v[:, 0], w[:, 0], u[0], torch.zeros(6, 4, dtype=F64))[0], P.wkv_scan(q, k, v, w, u)[:, 0])


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,dv,rot,halves", [(3, 12, 20, 8, True), (2, 64, 64, 64, True), (4, 4, 4, 0, True), (1, 128, 100, 32, False), (2, 32, 130, 30, True), (1, 200, 8, 200, True)])
def test_retention_from_a_saved_state(chunked, dtype, H, d, dv, rot, halves):
    """Portions of one token, of less than a chunk and of several chunks, at positions in the thousands, from states that
    are not zero; decays from fast to one."""
    lens, slots, past = [1, 37, 130, 5], [4, 1, 3, 0], [0, 17, 4000, 63]
    T = sum(lens)
    wide = rnd(T, H * (2 * d + dv), seed=1).to(DEV, dtype)
    q, k, v = wide[:, :H * d], wide[:, H * d:2 * H * d], wide[:, 2 * H * d:]
    decay = torch.tensor([1.0, 0.3, 0.99, 0.9375][:H])
    inv = rotary_frequencies(rot, 500.0) if rot else None
    state0 = rnd(6, H, d, dv, seed=50)
    state, out = state0.to(DEV).clone(), torch.full((T, H * dv), 9.0, device=DEV)
    scratch = None
    if chunked:
        assert K.recurrence_chunked_supported("retention", d)
        scratch = torch.full((K.recurrence_scratch_floats("retention", lens, H, d, dv),), 5.0, device=DEV)
    ((ctx, live),) = list(Steps([[n] for n in lens], slots, dtype, past))
    K.recurrence("retention", q, k, v, state, ctx.cu_seqlens, ctx.slots, lens, out, H, d, dv, scratch=scratch, decay=decay.to(DEV),
                 k_scale=d ** -0.5, positions=ctx.positions, inv_freq=inv.to(DEV) if rot else None, rot_dims=rot, half_layout=halves)
    r = 0
    freq = inv.double() if rot else torch.zeros(0, dtype=F64)
    for s, n in enumerate(lens):
        pos = torch.arange(past[s], past[s] + n)
        qq, kk = (P.rotate(t[r:r + n].double().cpu().view(n, H, d), pos, freq, halves) for t in (q, k))
        vv = v[r:r + n].double().cpu().view(n, H, dv)
        for h in range(H):
            o, S = walk_retention(qq[:, h], kk[:, h] * d ** -0.5, vv[:, h], float(decay[h]), state0[slots[s], h].double())
            close(out[r:r + n].view(n, H, dv)[:, h], o, torch.float32, f"sequence {s} head {h}", f32=3e-4)
            close(state[slots[s], h], S, torch.float32, "state", f32=3e-4)
        r += n
    assert torch.equal(state[[2, 5]].cpu(), state0[[2, 5]])


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,dv", [(3, 16, 16), (2, 64, 64), (1, 40, 24), (2, 128, 128), (1, 12, 70), (1, 172, 32)])
def test_time_mixing_recurrence_from_a_saved_state(chunked, dtype, H, d, dv):
    """Decays per channel and token from instant (exp(-exp(6))) to none (exp(-exp(-9))) side by side, a bonus that is far
    from one, portions of one token to several chunks."""
    lens, slots = [1, 37, 130, 16, 5], [4, 1, 3, 0, 2]
    T = sum(lens)
    wide = rnd(T, H * (2 * d + dv), seed=1).to(DEV, dtype)
    q, k, v = wide[:, :H * d], wide[:, H * d:2 * H * d], wide[:, 2 * H * d:]
    g = torch.Generator().manual_seed(8)
    a_bias = torch.rand(H * d, generator=g) * 12.0 - 9.0
    a, bonus = rnd(T, H * d, seed=3, scale=1.5), rnd(H * d, seed=4, scale=2.0)
    a[20, :] = 90.0      # a token after which nothing of the state is left
    state0 = rnd(6, H, d, dv, seed=50)
    state, out = state0.to(DEV).clone(), torch.full((T, H * dv), 9.0, device=DEV)
    scratch = None
    if chunked:
        assert K.recurrence_chunked_supported("wkv", d)
        scratch = torch.full((K.recurrence_scratch_floats("wkv", lens, H, d, dv),), 5.0, device=DEV)
    ((ctx, live),) = list(Steps([[n] for n in lens], slots, dtype))
    K.recurrence("wkv", q, k, v, state, ctx.cu_seqlens, ctx.slots, lens, out, H, d, dv, scratch=scratch, a=a.to(DEV),
                 a_bias=a_bias.to(DEV), bonus=bonus.to(DEV))
    w = torch.exp(-torch.exp(a.double() + a_bias.double())).view(T, H, d)
    r = 0
    for s, n in enumerate(lens):
        qq, kk, vv = (t[r:r + n].double().cpu().view(n, H, -1) for t in (q, k, v))
        for h in range(H):
            o, S = walk_wkv(qq[:, h], kk[:, h], vv[:, h], w[r:r + n, h], bonus.double().view(H, d)[h], state0[slots[s], h].double())
            close(out[r:r + n].view(n, H, dv)[:, h], o, torch.float32, f"sequence {s} head {h}", f32=3e-5)
            close(state[slots[s], h], S, torch.float32, "state", f32=3e-5)
        r += n
    assert torch.equal(state[5].cpu(), state0[5])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,vdim,rot", [(12, 20, 8), (10, 14, 6), (64, 64, 64)])
def test_retention_mixer_in_any_cut(dtype, dim, vdim, rot):
    D, decay, eps = 48, (0.5, 0.9, 0.99), 1e-3
    m = {"heads": 3, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": {"dims": rot, "base": 50.0}}
    W = {n: rnd(3 * r, D, seed=i, scale=0.3) for i, (n, r) in enumerate((("q", dim), ("k", dim), ("v", vdim), ("g", vdim)))}
    W["o"] = rnd(D, 3 * vdim, seed=8, scale=0.3)
    part = build_part("mixer", PartSpec("retention", "mix", {"heads": 3, "dim": dim, "vdim": vdim, "decay": decay, "norm_eps": eps,
                                                             "rot_dims": rot, "rot_base": 50.0}), hidden_size=D)
    part.bind({k: w.to(DEV, dtype) for k, w in W.items()})
    part.finalize(dtype, torch.device(DEV))
    x = [rnd(n, D, seed=40 + i) for i, n in enumerate(LENGTHS)]
    got = run_part(part, x, CUTS, SLOTS, dtype, 16, 4)
    for s, t in enumerate(x):
        want = P.retention(t.double(), {k: v.double() for k, v in W.items()}, "", m, eps, torch.arange(LENGTHS[s]))
        close(got[s], want, dtype, f"sequence {s}", f32=1e-4, bf16=3e-2)


# ----------------------------------------------------------------------------- time mixing
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,n_mixes", [(44, 5), (50, 3), (1024, 5), (2052, 8), (3, 1)])
def test_shifted_mixes_in_any_cut(dtype, D, n_mixes):
    x = [rnd(n, D, seed=i) for i, n in enumerate(LENGTHS)]
    mu = torch.rand(n_mixes, D, generator=torch.Generator().manual_seed(5)) * 1.6 - 0.3
    state = torch.full((7, D), 7.0, device=DEV)
    state[SLOTS] = 0.0
    for ctx, live in Steps(CUTS, SLOTS, dtype):
        rows = torch.cat([x[s][a:a + n] for s, a, n in live]).to(DEV, dtype)
        out = torch.full((n_mixes, ctx.n_tokens + 3, D), 9.0, dtype=dtype, device=DEV)
        K.shifted_mixes(rows, mu.to(DEV), state, ctx.cu_seqlens, ctx.slots, ctx.seq_of, out)
        for j in range(n_mixes):
            want = torch.cat([P.shifted_mix(x[s].double(), mu[j].double())[a:a + n] for s, a, n in live])
            close(out[j, :ctx.n_tokens], want, dtype, f"mix {j}", f32=1e-6, bf16=1e-2)
        assert float((out[:, ctx.n_tokens:].float() - 9.0).abs().max()) == 0.0
        for s, a, n in live:
            assert torch.equal(state[SLOTS[s]].cpu(), x[s][a + n - 1])
    assert torch.equal(state[1], torch.full_like(state[1], 7.0))


def test_shifted_mixes_of_a_long_step():
    """So many tokens that a block takes several rows: rows that start a sequence in the middle of a block's rows."""
    D, dtype, lens = 256, torch.bfloat16, [3001, 1, 2, 999, 1500]
    x, mu = rnd(sum(lens), D, seed=2), torch.rand(5, D)
    ((ctx, live),) = list(Steps([[n] for n in lens], [0, 1, 2, 3, 4], dtype))
    state0 = rnd(5, D, seed=3)
    state, out = state0.to(DEV).clone(), torch.empty(5, sum(lens), D, dtype=dtype, device=DEV)
    K.shifted_mixes(x.to(DEV, dtype), mu.to(DEV), state, ctx.cu_seqlens, ctx.slots, ctx.seq_of, out)
    r = 0
    for s, n in enumerate(lens):
        rows = x[r:r + n].double()
        before = torch.cat([state0[s:s + 1].double(), rows[:-1]])
        for j in range(5):
            close(out[j, r:r + n], rows + (before - rows) * mu[j].double(), dtype, f"sequence {s} mix {j}", bf16=1e-2)
        assert torch.equal(state[s].cpu(), x[r + n - 1])
        r += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,R,C", [(1, 5, 48), (8, 16, 100), (64, 64, 256), (77, 24, 33), (300, 128, 64), (3, 1000, 40)])
def test_low_rank_tanh_product(dtype, T, R, C):
    z, w = rnd(T, R + 2, seed=1, scale=1.5), rnd(C, R, seed=2, scale=R ** -0.5)
    out = torch.empty(T, C, device=DEV)
    zz = z.to(DEV, dtype)[:, 2:]
    K.low_rank_tanh(zz, w.to(DEV, dtype), out)
    close(out, torch.tanh(z[:, 2:].double()) @ w.double().t(), torch.float32, "low rank")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,H,dim,rank", [(48, 3, 16, 5), (50, 2, 12, 7), (128, 2, 64, 32), (64, 1, 100, 8)])
def test_time_mix_in_any_cut(dtype, D, H, dim, rank):
    """The whole mixer, with and without the weight-streaming products (by width), through steps that mix portions and
    single tokens; the bonus, the mixes and the decays show when changed in the oracle."""
    I, eps = H * dim, 1e-3
    g = torch.Generator().manual_seed(4)
    W = {f"mu.{s}": torch.rand(D, generator=g) * 1.4 - 0.2 for s in "rkvgw"}
    W.update({s: rnd(I, D, seed=i, scale=D ** -0.5 * 1.3) for i, s in enumerate("rkvg")})
    W.update({"w1": rnd(rank, D, seed=6, scale=D ** -0.5), "w2": rnd(I, rank, seed=7, scale=rank ** -0.5), "w0": torch.rand(I, generator=g) * 7 - 5.5,
              "u": rnd(H, dim, seed=8), "norm": rnd(I, seed=9) * 0.3 + 1.0, "o": rnd(D, I, seed=10, scale=I ** -0.5 * 1.3)})
    part = build_part("mixer", PartSpec("time_mix", "mix", {"heads": H, "dim": dim, "decay_rank": rank, "norm_eps": eps}), hidden_size=D)
    part.bind({ps.name: W[ps.name].to(DEV, dtype if ps.kind == "matrix" else torch.float32) for ps in part.param_specs()})
    part.finalize(dtype, torch.device(DEV))
    x = [rnd(n, D, seed=40 + i) for i, n in enumerate(LENGTHS)]
    W64, m = {k: v.double() for k, v in W.items()}, {"heads": H, "dim": dim}
    want = [P.wkv(t.double(), W64, "", m, eps) for t in x]
    for name, other in (("u", W64["u"] * 0), ("mu.w", W64["mu.w"] * 0), ("w0", W64["w0"] + 1.0), ("mu.r", W64["mu.r"] * 0)):
        assert float((P.wkv(x[0].double(), dict(W64, **{name: other}), "", m, eps) - want[0]).abs().max()) > 0.1, name
    got = run_part(part, x, CUTS, SLOTS, dtype, 16, 4)
    for s, ref in enumerate(want):
        close(got[s], ref, dtype, f"sequence {s}", f32=1e-4, bf16=4e-2)


# ----------------------------------------------------------------------------- parallel mixer, feed-forward
@pytest.mark.parametrize("dtype", DTYPES)
def test_the_two_sides_are_normed_and_halved(dtype):
    """The sides' results differ in size by far: a sum before the norms, or one weight for both, would show."""
    D, eps = 48, 1e-3
    m = {"left": {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.3, "mask": {"size": 24}},
         "right": {"heads": 2, "dim": 12, "vdim": 20, "decay": [0.6, 0.98], "rot": {"dims": 8, "base": 50.0}}}
    W = {"left.q": rnd(64, D, seed=1, scale=0.3), "left.k": rnd(32, D, seed=2, scale=0.3), "left.v": rnd(48, D, seed=3, scale=0.3),
         "left.o": rnd(D, 96, seed=4, scale=3.0), "left.out": rnd(D, seed=5) * 0.3 + 1.0, "right.out": rnd(D, seed=6) * 0.3 - 1.0,
         "right.q": rnd(24, D, seed=7, scale=0.3), "right.k": rnd(24, D, seed=8, scale=0.3), "right.v": rnd(40, D, seed=9, scale=0.3),
         "right.g": rnd(40, D, seed=10, scale=0.3), "right.o": rnd(D, 40, seed=11, scale=0.1)}
    l, r = m["left"], m["right"]
    part = build_part("mixer", PartSpec("normed_parallel", "mix", {"eps": eps, "scale": 0.5, "branches": [
        {"name": "left", "kind": "head_norm_attention", "params": {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.3, "norm_eps": eps,
                                                                   "chunk": 24, "one_more": True}},
        {"name": "right", "kind": "retention", "params": {"heads": 2, "dim": 12, "vdim": 20, "decay": r["decay"], "norm_eps": eps, "rot_dims": 8,
                                                          "rot_base": 50.0}}]}), hidden_size=D)
    part.bind({ps.name: W[ps.name].to(DEV, dtype if ps.kind == "matrix" else torch.float32) for ps in part.param_specs()})
    part.finalize(dtype, torch.device(DEV))
    x = [rnd(n, D, seed=40 + i) for i, n in enumerate(LENGTHS)]
    got = run_part(part, x, CUTS, SLOTS, dtype, 16, 24)
    for s, t in enumerate(x):
        want = P.parallel(t.double(), {k: v.double() for k, v in W.items()}, "", m, eps, torch.arange(LENGTHS[s]))
        close(got[s], want, dtype, f"sequence {s}", f32=1e-4, bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,D,F", [(1, 64, 96), (5, 50, 33), (16, 256, 512), (40, 1024, 320), (64, 2048, 64), (63, 96, 40), (300, 64, 88), (6000, 128, 1024)])
def test_plain_feed_forward_in_all_its_forms(dtype, T, D, F):
    """Weight-streaming products of up to 64 tokens in both tensor-core forms, and the library product with a launch for the
    activation; GELU's exact form (the tanh form differs by up to 5e-4)."""
    part = build_part("feed_forward", PartSpec("mlp", "mlp", {"intermediate_size": F, "activation": "gelu", "tensors": ("up", "down")}), hidden_size=D)
    up, down = rnd(F, D, seed=1, scale=1.5 * D ** -0.5), rnd(D, F, seed=2, scale=F ** -0.5)
    part.bind({"up": up.to(DEV, dtype), "down": down.to(DEV, dtype)})
    x = rnd(T, D, seed=3)
    ctx = StepContext(T, *([None] * 7), n_rows=0, decode_only=T == 1, kv_len_bound=1, dtype=dtype, workspace=Workspace(torch.device(DEV)))
    out = torch.empty(T, D, dtype=dtype, device=DEV)
    part.forward(x.to(DEV, dtype), ctx, out)
    K.check_status(torch.device(DEV), wait=True)
    want = P.feed_forward(x.double(), {"up": up.double(), "down": down.double()}, "")
    close(out, want, dtype, "feed-forward", bf16=1e-2)


def test_gelu_is_exact_where_the_tanh_form_is_not():
    z = torch.linspace(-6, 6, 4001)
    x = z.to(DEV).view(1, -1).clone()
    K.gelu_(x)
    close(x[0], P.gelu_erf(z.double()), torch.float32, "gelu", f32=1e-6)
    tanh_form = torch.nn.functional.gelu(z.double(), approximate="tanh")
    assert float((P.gelu_erf(z.double()) - tanh_form).abs().max()) > 1e-4
    zb = z.to(torch.bfloat16)     # the short form for bfloat16 results: within half a step of bfloat16 and 1e-6 of the exact one
    for width in (4000, 4001):    # eight elements a thread, and one by one
        y = zb[:width].to(DEV).view(1, -1).clone()
        K.gelu_(y)
        want = P.gelu_erf(zb[:width].double())
        assert bool(((y[0].double().cpu() - want).abs() <= want.abs() * 2.0 ** -8 + 1e-6).all())
    t = z.to(DEV).view(1, -1).clone()
    K.tanh_(t)
    close(t[0], torch.tanh(z.double()), torch.float32, "tanh", f32=1e-6)


@pytest.mark.parametrize("M", [1, 8, 13, 32, 64])
def test_several_products_in_one_launch(M):
    K_, ns = 200, [96, 40, 7, 1000, 33]
    xs = [rnd(M, K_, seed=i).to(DEV, torch.bfloat16) for i in range(5)]
    ws = [rnd(n, K_, seed=10 + n, scale=0.1).to(DEV, torch.bfloat16) for n in ns]
    outs = [torch.full((M, n + 3), 9.0, dtype=torch.bfloat16, device=DEV) for n in ns]
    K.skinny_linears(xs, ws, [o[:, :n] for o, n in zip(outs, ns)])
    for x, w, o, n in zip(xs, ws, outs, ns):
        close(o[:, :n], x.double().cpu() @ w.double().cpu().t(), torch.bfloat16, f"columns {n}", bf16=1e-2)
        assert float((o[:, n:].float() - 9.0).abs().max()) == 0.0
