// The selective scan with a decay per channel and state entry (Mamba-1):
//
//   dt_c = softplus(raw_c + bias_c),  A[c, n] = -exp(A_log[c, n])
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = (sum_n S[c, n] C_n + D_c x_c) * silu(z_c)
//
// B and C [N] belong to the token, S [slots][I][N] float to the request.  The decay differs for every state entry,
// so there is no matrix form: the work is one exponential and four multiply-adds per (token, channel, entry), and
// the exponential unit (16 lanes a clock and SM) is the bound of prompt steps.
//
// A block owns 128 / LN channels of one chunk and has two halves of four warps.  In the walking half LN neighbouring lanes
// share a channel and keep NPT state entries each in registers for the whole walk (LN * NPT >= N; entries beyond N have
// B = C = 0): a token costs a lane two shared-memory reads and five instructions an entry, and nothing but the
// state's own multiply-add waits for the token before.  The other half runs beside it, one tile of tokens ahead and one
// behind: it widens the next tile's B and C, makes its step sizes and dt * x, requests the tile after that, and gates
// and writes the outputs of the tile before.  One barrier a tile; the tiles' shared memory has two places.
//
// Portions are cut into chunks only where one walk per channel would leave most of the GPU empty:
//   chunk_state   every chunk but a sequence's last, from a zero state: its end state and the sum of its dt
//   chunk_pass    per state entry, over the chunks of a sequence: the chunks' start states
//   walk          every chunk from its start state, with the outputs
// (two exponentials per entry instead of one); else the walk starts from the request's state.  The float storage
// type walks in double, unchunked.  One token per sequence (decode): selective_step, which also makes the channel's
// raw step size from the low-rank row, raw_c = W_dt[c] . low[:R], unless it is given.
#include "common.cuh"
#include <type_traits>

namespace pmm {

constexpr int kSelThreads = 128;
constexpr int kSelWalkThreads = 2 * kSelThreads;  // the walking half and the half that makes its inputs

// Base-2 exponential: the walk multiplies A by log2(e) once.  Approximate to 2 ulp in float.
__device__ __forceinline__ float sel_exp2(float v) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}
__device__ __forceinline__ double sel_exp2(double v) { return exp2(v); }

// NPT neighbouring state entries from n0 on (0 beyond N); whole 16-byte pieces where `vec` says that N is a multiple of 4.
template <int NPT>
__device__ __forceinline__ void sel_ld_state(const float* row, int n0, int N, bool vec, float* o) {
  if (NPT % 4 == 0 && vec) {
#pragma unroll
    for (int i = 0; i < NPT; i += 4) {
      const float4 v = n0 + i < N ? *reinterpret_cast<const float4*>(row + n0 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      o[i] = v.x; o[i + 1] = v.y; o[i + 2] = v.z; o[i + 3] = v.w;
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < NPT; ++i) o[i] = n0 + i < N ? row[n0 + i] : 0.f;
}
template <int NPT>
__device__ __forceinline__ void sel_st_state(float* row, int n0, int N, bool vec, const float* o) {
  if (NPT % 4 == 0 && vec) {
#pragma unroll
    for (int i = 0; i < NPT; i += 4)
      if (n0 + i < N) *reinterpret_cast<float4*>(row + n0 + i) = make_float4(o[i], o[i + 1], o[i + 2], o[i + 3]);
    return;
  }
#pragma unroll
  for (int i = 0; i < NPT; ++i)
    if (n0 + i < N) row[n0 + i] = o[i];
}
struct SelArgs {
  const void* x;        // [T, I] after convolution and activation, rows of ld_x
  const void* raw;      // [T, I] step sizes before bias and softplus
  const void* low;      // [T, ...]: B at column off_b, C at off_c (decode: the low-rank row at column 0)
  const void* z;        // [T, I] gate
  long long ld_x, ld_raw, ld_low, ld_z;
  int off_b, off_c;
  const float* bias;    // [I]
  const float* a_log;   // [I, N]
  const float* d;       // [I]
  float* state;         // [slots, I, N]
  float* chunk_state;   // [chunks, I, N]: end states, then start states
  float* chunk_dt;      // [chunks, I]
  const int* cu;
  const int* slots;
  void* y;              // [T, I]
  int n_seq, I, N, chunk_len;
  const void* w_dt;     // decode: [I, R]
  int R;
  int pairs;            // rows of x, raw, z and y may be read two channels at a time
  int bc_pairs;         // B and C two entries at a time
};

// The sequence and the chunk within it of global chunk `idx`; false when there is no such chunk.  Called by whole warps.
__device__ __forceinline__ bool sel_find_chunk(const int* __restrict__ cu, int n_seq, int chunk_len, int idx, int* seq, int* k,
                                               int* n_chunks) {
  const int lane = threadIdx.x & 31;
  int before = 0;
  for (int s0 = 0; s0 < n_seq; s0 += 32) {
    const int s = s0 + lane;
    const int n = s < n_seq ? cu[s + 1] - cu[s] : 0;
    const int mine = (n + chunk_len - 1) / chunk_len;
    int incl = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += v;
    }
    const int lo = before + incl - mine;
    const unsigned hit = __ballot_sync(0xffffffffu, idx >= lo && idx < lo + mine);
    if (hit) {
      const int src = __ffs(hit) - 1;
      *seq = s0 + src;
      *k = idx - __shfl_sync(0xffffffffu, lo, src);
      *n_chunks = __shfl_sync(0xffffffffu, mine, src);
      return true;
    }
    before += __shfl_sync(0xffffffffu, incl, 31);
  }
  return false;
}

// A thread's two neighbouring channels of one token as they lie in memory.
template <typename S>
struct SelPair;
template <>
struct SelPair<__nv_bfloat16> {
  __nv_bfloat162 v;
  __device__ __forceinline__ float2 get() const { return __bfloat1622float2(v); }
};
template <>
struct SelPair<float> {
  float2 v;
  __device__ __forceinline__ float2 get() const { return v; }
};
__device__ __forceinline__ void sel_ld_pair(const __nv_bfloat16* p, bool whole, bool second, SelPair<__nv_bfloat16>& o) {
  if (whole) {
    o.v = *reinterpret_cast<const __nv_bfloat162*>(p);
  } else {
    o.v.x = p[0];
    o.v.y = second ? p[1] : __float2bfloat16_rn(0.f);
  }
}
__device__ __forceinline__ void sel_ld_pair(const float* p, bool, bool second, SelPair<float>& o) {
  o.v.x = p[0];
  o.v.y = second ? p[1] : 0.f;
}
__device__ __forceinline__ void sel_zero(SelPair<__nv_bfloat16>& o) { o.v = __floats2bfloat162_rn(0.f, 0.f); }
__device__ __forceinline__ void sel_zero(SelPair<float>& o) { o.v = make_float2(0.f, 0.f); }

// softplus(v) = max(v, 0) + log(1 + e), e = exp(-|v|).  Float: base-2 approximations; where e is small, 1 + e would round
// it away, so the series of log(1 + e) takes over (below 1/16 its fifth term is under 2e-7 of the sum).
__device__ __forceinline__ float sel_softplus(float v) {
  const float e = sel_exp2(-1.4426950408889634f * fabsf(v));
  float lg;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(lg) : "f"(1.f + e));
  const float series = e * (1.f - e * (0.5f - e * (1.f / 3.f - e * (0.25f - e * 0.2f))));
  return fmaxf(v, 0.f) + (e < 0.0625f ? series : 0.6931471805599453f * lg);
}
__device__ __forceinline__ double sel_softplus(double v) { return scan_softplus<double>(v); }

template <typename ACC>
struct SelDu {
  ACC dt, u;
};

__device__ __forceinline__ void sel_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(kSelWalkThreads) : "memory"); }

// Tokens per tile for NB state entries of a channel (padded).
template <typename ACC, int NB>
struct SelTile {
  static constexpr int kFloat = NB <= 32 ? 32 : NB <= 128 ? 16 : 8;
  static constexpr int kTokens = sizeof(ACC) == 8 && kFloat > 16 ? 16 : kFloat;
};

// OUT: the walk with outputs.  Otherwise chunk_state.  A lane's entries are pairs: entry (i * LN + q) * 2 + j.
template <typename S, typename ACC, int LN, int NPT, bool OUT>
__global__ void __launch_bounds__(kSelWalkThreads, sizeof(ACC) == 4 ? 3 : 2) selective_walk_kernel(const SelArgs p) {
  constexpr int CH = kSelThreads / LN, NB = LN * NPT, NP = NPT / 2;
  constexpr int TT = SelTile<ACC, NB>::kTokens;
  constexpr int G = LN < 8 ? LN : 8;   // tokens whose sums over the lanes are made together
  __shared__ __align__(16) SelDu<ACC> s_du[2][TT][CH];
  __shared__ __align__(16) float2 s_bc[2][TT][NB];  // (B, C) of an entry
  __shared__ ACC s_y[2][OUT ? TT : 1][CH];
  pdl_launch_dependents();
  const bool walker = threadIdx.x < kSelThreads;
  const int tid = threadIdx.x % kSelThreads;
  const int c0 = blockIdx.x * CH;
  const int N = p.N, I = p.I;
  pdl_wait();
  int seq, k, n_chunks;
  if (!sel_find_chunk(p.cu, p.n_seq, p.chunk_len, blockIdx.y, &seq, &k, &n_chunks)) return;
  if (!OUT && k == n_chunks - 1) return;  // nobody starts from a sequence's last chunk
  const int t_end = p.cu[seq + 1];
  const int t0 = p.cu[seq] + k * p.chunk_len, t1 = min(t_end, t0 + p.chunk_len);
  const int n_tiles = (t1 - t0 + TT - 1) / TT;

  if (walker) {
    const int ch = tid / LN, q = tid % LN, c = c0 + ch;
    const bool ok = c < I;
    const bool even = N % 2 == 0;
    float* slot_state = p.state + (static_cast<size_t>(p.slots[seq]) * I + (ok ? c : 0)) * N;
    float* mine = n_chunks > 1 ? p.chunk_state + (static_cast<size_t>(blockIdx.y) * I + (ok ? c : 0)) * N : slot_state;
    const float* al = p.a_log + static_cast<size_t>(ok ? c : 0) * N;
    ACC a2[NPT], st[NPT];
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int n = (i * LN + q) * 2;
      float2 av = make_float2(0.f, 0.f), sv = make_float2(0.f, 0.f);
      if (n < N && even) {
        av = *reinterpret_cast<const float2*>(al + n);
        if (OUT) sv = *reinterpret_cast<const float2*>(mine + n);
      } else if (n < N) {
        av = make_float2(al[n], n + 1 < N ? al[n + 1] : 0.f);
        if (OUT) sv = make_float2(mine[n], n + 1 < N ? mine[n + 1] : 0.f);
      }
      a2[2 * i] = static_cast<ACC>(-1.4426950408889634) * scan_exp(static_cast<ACC>(av.x));
      a2[2 * i + 1] = static_cast<ACC>(-1.4426950408889634) * scan_exp(static_cast<ACC>(av.y));
      st[2 * i] = sv.x;
      st[2 * i + 1] = sv.y;
    }
    ACC dt_sum = 0;
    sel_barrier();
    for (int tile = 0; tile < n_tiles; ++tile) {
      const int buf = tile & 1;
#pragma unroll
      for (int g = 0; g < TT; g += G) {
        ACC acc[G];
#pragma unroll
        for (int j = 0; j < G; ++j) {
          const SelDu<ACC> du = s_du[buf][g + j][ch];
          ACC sum = 0;
#pragma unroll
          for (int i = 0; i < NP; ++i) {
            const float4 bc = *reinterpret_cast<const float4*>(&s_bc[buf][g + j][(i * LN + q) * 2]);
            st[2 * i] = sel_exp2(du.dt * a2[2 * i]) * st[2 * i] + du.u * static_cast<ACC>(bc.x);
            st[2 * i + 1] = sel_exp2(du.dt * a2[2 * i + 1]) * st[2 * i + 1] + du.u * static_cast<ACC>(bc.z);
            if (OUT) {
              sum += st[2 * i] * static_cast<ACC>(bc.y);
              sum += st[2 * i + 1] * static_cast<ACC>(bc.w);
            }
          }
          acc[j] = sum;
          if (!OUT) dt_sum += du.dt;
        }
        if (OUT) {
          // the lanes' sums of G tokens: at every level a lane hands half of its tokens to its partner and keeps the
          // other half, so that lane q ends with the whole sum of token q
#pragma unroll
          for (int o = G / 2; o > 0; o >>= 1) {
            const bool up = (q & o) != 0;
#pragma unroll
            for (int j = 0; j < o; ++j) {
              const ACC send = up ? acc[j] : acc[j + o];
              const ACC keep = up ? acc[j + o] : acc[j];
              acc[j] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
          }
#pragma unroll
          for (int o = G; o < LN; o <<= 1) acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], o);
          if (q < G) s_y[buf][OUT ? g + q : 0][ch] = acc[0];
        }
      }
      sel_barrier();
    }
    if (!ok) return;
    float* dst = OUT ? slot_state : mine;
    if (!OUT || k == n_chunks - 1) {
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int n = (i * LN + q) * 2;
        if (n < N && even) {
          *reinterpret_cast<float2*>(dst + n) = make_float2(static_cast<float>(st[2 * i]), static_cast<float>(st[2 * i + 1]));
        } else if (n < N) {
          dst[n] = static_cast<float>(st[2 * i]);
          if (n + 1 < N) dst[n + 1] = static_cast<float>(st[2 * i + 1]);
        }
      }
    }
    if (!OUT && q == 0) p.chunk_dt[static_cast<size_t>(blockIdx.y) * I + c] = static_cast<float>(dt_sum);
    return;
  }

  // ------------------------------------------------------------------ the other half: thread -> (token of the tile, pair of channels)
  constexpr int HC = CH / 2;
  constexpr int PX = (TT * HC + kSelThreads - 1) / kSelThreads;
  constexpr int TSTEP = kSelThreads / HC;                          // tokens between a thread's pairs
  constexpr int HB = NB / 2;
  constexpr int PB = (TT * HB + kSelThreads - 1) / kSelThreads;    // (token, pair of entries) per thread
  const int tt0 = tid / HC, cp = (tid % HC) * 2, cc = c0 + cp;
  const bool in0 = cc < I && tt0 < TT, in1 = cc + 1 < I;
  const float bias0 = in0 ? p.bias[cc] : 0.f, bias1 = in0 && in1 ? p.bias[cc + 1] : 0.f;
  const float d0 = (OUT && in0) ? p.d[cc] : 0.f, d1 = (OUT && in0 && in1) ? p.d[cc + 1] : 0.f;
  SelPair<S> rx[PX], rd[PX], rz[OUT ? PX : 1];      // the next tile as it lies in memory
  SelPair<S> rb[PB], rc[PB];
  SelPair<S> xw[OUT ? PX : 1], zw[OUT ? PX : 1];    // x and z of the tile that is walked
  SelPair<S> xg[OUT ? PX : 1], zg[OUT ? PX : 1];    // ... and of the one before it
  const bool whole = in1 && p.pairs, bwhole = p.bc_pairs != 0;
  const S* xs = static_cast<const S*>(p.x) + static_cast<long long>(t0 + tt0) * p.ld_x + (in0 ? cc : 0);
  const S* ds = static_cast<const S*>(p.raw) + static_cast<long long>(t0 + tt0) * p.ld_raw + (in0 ? cc : 0);
  const S* zs = OUT ? static_cast<const S*>(p.z) + static_cast<long long>(t0 + tt0) * p.ld_z + (in0 ? cc : 0) : nullptr;
  const S* ls = static_cast<const S*>(p.low) + static_cast<long long>(t0) * p.ld_low;
  auto request = [&](int tile) {
    const int left = t1 - t0 - tile * TT;  // the chunk's tokens from the tile's first on
#pragma unroll
    for (int r = 0; r < PX; ++r) {
      if (in0 && tt0 + r * TSTEP < left) {
        sel_ld_pair(xs + r * TSTEP * p.ld_x, whole, in1, rx[r]);
        sel_ld_pair(ds + r * TSTEP * p.ld_raw, whole, in1, rd[r]);
        if (OUT) sel_ld_pair(zs + r * TSTEP * p.ld_z, whole, in1, rz[OUT ? r : 0]);
      } else {
        sel_zero(rx[r]);
        sel_zero(rd[r]);
        if (OUT) sel_zero(rz[OUT ? r : 0]);
      }
    }
#pragma unroll
    for (int r = 0; r < PB; ++r) {
      const int e = r * kSelThreads + tid, tt = e / HB, n = (e % HB) * 2;
      if (tt < TT && tt < left && n < N) {
        const S* row = ls + tt * p.ld_low + n;
        sel_ld_pair(row + p.off_b, bwhole, n + 1 < N, rb[r]);
        if (OUT) sel_ld_pair(row + p.off_c, bwhole, n + 1 < N, rc[r]);
      } else {
        sel_zero(rb[r]);
        if (OUT) sel_zero(rc[r]);
      }
      if (!OUT) sel_zero(rc[r]);
    }
    xs += TT * p.ld_x;
    ds += TT * p.ld_raw;
    if (OUT) zs += TT * p.ld_z;
    ls += TT * p.ld_low;
  };
  auto stage = [&](int tile) {
    const int buf = tile & 1, left = t1 - t0 - tile * TT;
#pragma unroll
    for (int r = 0; r < PX; ++r) {
      const int tt = tt0 + r * TSTEP;
      if (OUT) {
        xg[OUT ? r : 0] = xw[OUT ? r : 0];
        zg[OUT ? r : 0] = zw[OUT ? r : 0];
        xw[OUT ? r : 0] = rx[r];
        zw[OUT ? r : 0] = rz[OUT ? r : 0];
      }
      if (TT * HC < kSelThreads && tt >= TT) continue;
      const float2 x = rx[r].get(), raw = rd[r].get();
      // (tokens past the chunk's end: dt = 0 leaves the state as it is)
      const ACC dt0 = tt < left ? sel_softplus(static_cast<ACC>(raw.x) + static_cast<ACC>(bias0)) : static_cast<ACC>(0);
      const ACC dt1 = tt < left ? sel_softplus(static_cast<ACC>(raw.y) + static_cast<ACC>(bias1)) : static_cast<ACC>(0);
      s_du[buf][tt][cp] = {dt0, dt0 * static_cast<ACC>(x.x)};
      s_du[buf][tt][cp + 1] = {dt1, dt1 * static_cast<ACC>(x.y)};
    }
#pragma unroll
    for (int r = 0; r < PB; ++r) {
      const int e = r * kSelThreads + tid, tt = e / HB, n = (e % HB) * 2;
      if (tt < TT) {
        const float2 b = rb[r].get(), c = rc[r].get();
        *reinterpret_cast<float4*>(&s_bc[buf][tt][n]) = make_float4(b.x, c.x, b.y, c.y);
      }
    }
  };
  auto finish = [&](int tile, const SelPair<S>* xr, const SelPair<S>* zr) {  // the tile's outputs
    const int buf = tile & 1, base = t0 + tile * TT;
#pragma unroll
    for (int r = 0; r < PX; ++r) {
      const int tt = tt0 + r * TSTEP;
      if (!in0 || base + tt >= t1 || tt >= TT) continue;
      const float2 x = xr[r].get(), z = zr[r].get();
      const ACC y0 = static_cast<ACC>(d0) * static_cast<ACC>(x.x) + s_y[buf][OUT ? tt : 0][cp];
      const ACC y1 = static_cast<ACC>(d1) * static_cast<ACC>(x.y) + s_y[buf][OUT ? tt : 0][cp + 1];
      const float o0 = static_cast<float>(y0) * (sizeof(S) == 2 ? silu_fast(z.x) : silu_f(z.x));
      const float o1 = static_cast<float>(y1) * (sizeof(S) == 2 ? silu_fast(z.y) : silu_f(z.y));
      S* dst = static_cast<S*>(p.y) + static_cast<size_t>(base + tt) * I + cc;
      if (sizeof(S) == 2 && whole) {
        *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(o0, o1);
      } else {
        stf(dst, o0);
        if (in1) stf(dst + 1, o1);
      }
    }
  };
  request(0);
  stage(0);
  request(1);
  sel_barrier();
  for (int tile = 0; tile < n_tiles; ++tile) {
    if (OUT && tile > 0) finish(tile - 1, xg, zg);
    if (tile + 1 < n_tiles) {
      stage(tile + 1);  // (what is walked now becomes xg, zg)
      request(tile + 2);
    }
    sel_barrier();
  }
  if (OUT) finish(n_tiles - 1, xw, zw);
}

// A thread per state entry of a sequence of several chunks: chunk_state becomes the chunks' start states.
__global__ void __launch_bounds__(256) selective_chunk_pass_kernel(const SelArgs p) {
  pdl_launch_dependents();
  const int s = blockIdx.y;
  const int idx = blockIdx.x * blockDim.x + threadIdx.x;
  const bool ok = idx < p.I * p.N;
  const float a2 = ok ? -1.4426950408889634f * expf(p.a_log[idx]) : 0.f;
  pdl_wait();
  int first = 0;
  for (int i = 0; i < s; ++i) first += (p.cu[i + 1] - p.cu[i] + p.chunk_len - 1) / p.chunk_len;
  const int n_chunks = (p.cu[s + 1] - p.cu[s] + p.chunk_len - 1) / p.chunk_len;
  if (n_chunks < 2 || !ok) return;
  const int c = idx / p.N;
  const size_t stride = static_cast<size_t>(p.I) * p.N;
  float v = p.state[static_cast<size_t>(p.slots[s]) * stride + idx];
  float* cs = p.chunk_state + first * stride + idx;
  const float* cd = p.chunk_dt + static_cast<size_t>(first) * p.I + c;
#pragma unroll 4
  for (int k = 0; k < n_chunks; ++k) {
    const bool more = k + 1 < n_chunks;
    const float local = more ? cs[k * stride] : 0.f;
    const float dt = more ? cd[static_cast<size_t>(k) * p.I] : 0.f;
    cs[k * stride] = v;
    v = sel_exp2(dt * a2) * v + local;
  }
}

__device__ __forceinline__ void sel_ld8(const __nv_bfloat16* p, float* o) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    o[2 * i] = f.x;
    o[2 * i + 1] = f.y;
  }
}
// NPT neighbouring entries of B or C of a token (0 beyond N); vec: N a multiple of 4, pieces of 4 aligned.
template <int NPT>
__device__ __forceinline__ void sel_ld_row(const __nv_bfloat16* row, int n0, int N, bool vec, float* o) {
  if (NPT % 4 == 0 && vec) {
#pragma unroll
    for (int i = 0; i < NPT; i += 4) {
      uint2 raw = make_uint2(0u, 0u);
      if (n0 + i < N) raw = *reinterpret_cast<const uint2*>(row + n0 + i);
      const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
      const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
      o[i] = a.x; o[i + 1] = a.y; o[i + 2] = b.x; o[i + 3] = b.y;
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < NPT; ++i) o[i] = n0 + i < N ? __bfloat162float(row[n0 + i]) : 0.f;
}
template <int NPT>
__device__ __forceinline__ void sel_ld_row(const float* row, int n0, int N, bool, float* o) {
#pragma unroll
  for (int i = 0; i < NPT; ++i) o[i] = n0 + i < N ? row[n0 + i] : 0.f;
}
__device__ __forceinline__ void sel_ld8(const float* p, float* o) {
#pragma unroll
  for (int i = 0; i < 8; ++i) o[i] = p[i];
}

// One token per sequence: token s of sequence s.  vec: rows of low and W_dt in whole pieces of 8 elements.  (A block for
// several sequences, which would read the channel's constants once for all of them, was slower: 20 us for two and 27
// for four against 17, at 64 sequences of 6,144 channels.)
template <typename S, typename ACC, int LN, int NPT>
__global__ void __launch_bounds__(kSelThreads) selective_step_kernel(const SelArgs p, int vec) {
  constexpr int CH = kSelThreads / LN;
  pdl_launch_dependents();
  const int ch = threadIdx.x / LN, q = threadIdx.x % LN;
  const int c = blockIdx.x * CH + ch, s = blockIdx.y;
  const int N = p.N, I = p.I;
  const bool ok = c < I, svec = N % 4 == 0;
  const int cs = ok ? c : 0, n0 = q * NPT;
  ACC a2[NPT];
  {
    float al[NPT];
    sel_ld_state<NPT>(p.a_log + static_cast<size_t>(cs) * N, n0, N, svec, al);
#pragma unroll
    for (int i = 0; i < NPT; ++i) a2[i] = static_cast<ACC>(-1.4426950408889634) * scan_exp(static_cast<ACC>(al[i]));
  }
  const ACC bias = p.bias[cs], dskip = p.d[cs];
  float* srow = p.state + (static_cast<size_t>(p.slots[s]) * I + cs) * N;
  pdl_wait();
  float st[NPT], bv[NPT], cv[NPT];
  sel_ld_state<NPT>(srow, n0, N, svec, st);
  const S* low = static_cast<const S*>(p.low) + static_cast<long long>(s) * p.ld_low;
  const bool bvec = svec && vec && p.off_b % 4 == 0 && p.off_c % 4 == 0;
  sel_ld_row<NPT>(low + p.off_b, n0, N, bvec, bv);
  sel_ld_row<NPT>(low + p.off_c, n0, N, bvec, cv);
  const ACC xv = ldf(static_cast<const S*>(p.x) + static_cast<long long>(s) * p.ld_x + cs);
  const float zv = ldf(static_cast<const S*>(p.z) + static_cast<long long>(s) * p.ld_z + cs);
  ACC raw = 0;
  if (p.raw) {
    raw = ldf(static_cast<const S*>(p.raw) + static_cast<long long>(s) * p.ld_raw + cs);
  } else {
    const S* w = static_cast<const S*>(p.w_dt) + static_cast<size_t>(cs) * p.R;
    if (vec) {
      for (int r = q * 8; r < p.R; r += LN * 8) {
        float wv[8], lv[8];
        sel_ld8(w + r, wv);
        sel_ld8(low + r, lv);
#pragma unroll
        for (int i = 0; i < 8; ++i) raw += static_cast<ACC>(lv[i]) * static_cast<ACC>(wv[i]);
      }
    } else {
      for (int r = q; r < p.R; r += LN) raw += static_cast<ACC>(ldf(low + r)) * static_cast<ACC>(ldf(w + r));
    }
#pragma unroll
    for (int o = LN / 2; o > 0; o >>= 1) raw += __shfl_xor_sync(0xffffffffu, raw, o);
  }
  const ACC dt = sel_softplus(raw + bias);
  const ACC u = dt * xv;
  ACC acc = 0;
#pragma unroll
  for (int i = 0; i < NPT; ++i) {
    const ACC v = sel_exp2(dt * a2[i]) * static_cast<ACC>(st[i]) + u * static_cast<ACC>(bv[i]);
    acc += v * static_cast<ACC>(cv[i]);
    st[i] = static_cast<float>(v);
  }
#pragma unroll
  for (int o = LN / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
  if (!ok) return;
  sel_st_state<NPT>(srow, n0, N, svec, st);
  if (q == 0) stf(static_cast<S*>(p.y) + static_cast<size_t>(s) * I + c, static_cast<float>(acc + dskip * xv) * silu_f(zv));
}

// Lanes per channel of the walk for N state entries.
inline int sel_walk_lanes(int N) { return N <= 8 ? 4 : N <= 32 ? 8 : 16; }

template <typename S, bool OUT>
int launch_selective_walk(const SelArgs& p, int n_chunks, cudaStream_t stream) {
  using ACC = typename std::conditional<sizeof(S) == 4, double, float>::type;
  const int ch = kSelThreads / sel_walk_lanes(p.N);
  dim3 grid((p.I + ch - 1) / ch, n_chunks);
  // (no programmatic launch: blocks that start while the kernel before still holds part of the GPU pile up on the SMs it
  // has left, and this kernel lives from one long walk per SM)
#define PMM_SEL_WALK(LN, NPT) selective_walk_kernel<S, ACC, LN, NPT, OUT><<<grid, kSelWalkThreads, 0, stream>>>(p)
  if (p.N <= 8) PMM_SEL_WALK(4, 2);
  else if (p.N <= 16) PMM_SEL_WALK(8, 2);
  else if (p.N <= 32) PMM_SEL_WALK(8, 4);
  else if (p.N <= 64) PMM_SEL_WALK(16, 4);
  else if (p.N <= 128) PMM_SEL_WALK(16, 8);
  else PMM_SEL_WALK(16, 16);
#undef PMM_SEL_WALK
  return launch_status();
}

// Lanes per channel and entries per lane of the single step.
#define PMM_SEL_DISPATCH(N, CALL)      \
  do {                                 \
    if ((N) <= 4) { CALL(4, 1); }      \
    else if ((N) <= 8) { CALL(4, 2); } \
    else if ((N) <= 16) { CALL(4, 4); } \
    else if ((N) <= 32) { CALL(8, 4); } \
    else if ((N) <= 64) { CALL(16, 4); } \
    else if ((N) <= 128) { CALL(16, 8); } \
    else { CALL(16, 16); }             \
  } while (0)

inline int sel_lanes(int N) { return N <= 16 ? 4 : N <= 32 ? 8 : 16; }

template <typename S>
int launch_selective_step(const SelArgs& p, int vec, cudaStream_t stream) {
  using ACC = typename std::conditional<sizeof(S) == 4, double, float>::type;
  const int ch = kSelThreads / sel_lanes(p.N);
  dim3 grid((p.I + ch - 1) / ch, p.n_seq);
#define PMM_SEL_STEP(LN, NPT) launch_pdl(selective_step_kernel<S, ACC, LN, NPT>, grid, dim3(kSelThreads), 0, stream, p, vec)
  PMM_SEL_DISPATCH(p.N, PMM_SEL_STEP);
#undef PMM_SEL_STEP
  return launch_status();
}

}  // namespace pmm

// Channels of one block of the walk (for the host's choice of chunks).
PMM_EXPORT int pmm_selective_scan_channels(int N) { return N <= 0 || N > 256 ? 0 : pmm::kSelThreads / pmm::sel_walk_lanes(N); }

// x, raw, z [T, I] and low (B at off_b, C at off_c) in the storage type, unit column stride; y [T, I] contiguous.  n_chunks: at least
// sum over the sequences of ceil(tokens / chunk_len).  multi: some sequence may have more than one chunk (then chunk_state
// [n_chunks, I, N] and chunk_dt [n_chunks, I] floats; float storage has to go unchunked: chunk_len at least the longest portion).
PMM_EXPORT int pmm_selective_scan(const void* x, long long ld_x, const void* raw, long long ld_raw, const void* low,
                                  long long ld_low, int off_b, int off_c, const void* z, long long ld_z, const float* bias,
                                  const float* a_log, const float* d, float* state, float* chunk_state, float* chunk_dt,
                                  const int* cu, const int* slots, void* y, int n_seq, int n_chunks, int chunk_len, int multi,
                                  int I, int N, int dtype, cudaStream_t stream) {
  if (n_seq <= 0 || n_chunks <= 0) return 0;
  if (I <= 0 || N <= 0 || N > 256 || chunk_len <= 0 || n_chunks > 65535 || n_seq > 65535) return PMM_ERR_BAD_ARGUMENT;
  if (multi && (!chunk_state || !chunk_dt || dtype != PMM_DTYPE_BF16)) return PMM_ERR_BAD_ARGUMENT;
  pmm::SelArgs p{x, raw, low, z, ld_x, ld_raw, ld_low, ld_z, off_b, off_c, bias, a_log, d, state, chunk_state, chunk_dt, cu,
                 slots, y, n_seq, I, N, chunk_len, nullptr, 0, 0, 0};
  auto even = [&](const void* q, long long ld) { return reinterpret_cast<uintptr_t>(q) % 4 == 0 && ld % 2 == 0; };
  p.pairs = even(x, ld_x) && even(raw, ld_raw) && even(z, ld_z) && even(y, I);
  p.bc_pairs = even(low, ld_low) && off_b % 2 == 0 && off_c % 2 == 0 && N % 2 == 0;
  if (multi) {
    int rc = pmm::launch_selective_walk<__nv_bfloat16, false>(p, n_chunks, stream);
    if (rc != 0) return rc;
    pmm::launch_pdl(pmm::selective_chunk_pass_kernel, dim3((I * N + 255) / 256, n_seq), dim3(256), 0, stream, p);
    rc = pmm::launch_status();
    if (rc != 0) return rc;
  }
  PMM_DISPATCH_DTYPE(dtype, S, { return (pmm::launch_selective_walk<S, true>(p, n_chunks, stream)); });
  return 0;
}

// One token per sequence.  low [n_seq, ...]: the low-rank row of the step sizes in columns 0 .. R - 1, B at off_b, C at off_c;
// w_dt [I, R] contiguous.  raw [n_seq, I]: the raw step sizes, made already (w_dt and R are then not used); or nullptr.
PMM_EXPORT int pmm_selective_step(const void* x, long long ld_x, const void* raw, long long ld_raw, const void* low, long long ld_low, int R, int off_b, int off_c,
                                  const void* w_dt, const void* z, long long ld_z, const float* bias, const float* a_log,
                                  const float* d, float* state, const int* slots, void* y, int n_seq, int I, int N, int dtype,
                                  cudaStream_t stream) {
  if (n_seq <= 0) return 0;
  if (I <= 0 || N <= 0 || N > 256 || (!raw && (R <= 0 || !w_dt)) || n_seq > 65535) return PMM_ERR_BAD_ARGUMENT;
  pmm::SelArgs p{x, raw, low, z, ld_x, ld_raw, ld_low, ld_z, off_b, off_c, bias, a_log, d, state, nullptr, nullptr, nullptr,
                 slots, y, n_seq, I, N, 0, w_dt, R, 0, 0};
  const int vec = R % 8 == 0 && ld_low % 8 == 0 && reinterpret_cast<uintptr_t>(low) % 16 == 0 && reinterpret_cast<uintptr_t>(w_dt) % 16 == 0;
  PMM_DISPATCH_DTYPE(dtype, S, return pmm::launch_selective_step<S>(p, vec, stream));
  return 0;
}
