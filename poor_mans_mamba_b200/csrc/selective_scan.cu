// The selective scan with a decay per channel and state entry (Mamba-1):
//
//   dt_c = softplus(raw_c + bias_c),  A[c, n] = -exp(A_log[c, n])
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = (sum_n S[c, n] C_n + D_c x_c) * silu(z_c)
//
// B and C [N] belong to the token, S [slots][I][N] float to the request.  The decay differs for every state entry,
// so there is no matrix form: the work is one exponential and four multiply-adds per (token, channel, entry), and
// the exponential unit (16 lanes a clock and SM) is the bound of prompt steps.
//
// LN neighbouring lanes share a channel and keep NPT entries each in registers for the whole walk (LN * NPT >= N;
// entries beyond N have B = C = 0).  A block of 128 threads owns CH = 128 / LN channels of one chunk.  Tokens come
// through shared memory in tiles of kTile: every thread makes the softplus and dt * x of its share of the tile
// once, B and C are widened once, and the outputs of a tile are gated and written together.  The next tile's rows
// are requested before a tile is walked.
//
// Prompt portions are cut into chunks only where one walk per channel would leave the GPU empty:
//   chunk_state   every chunk but a sequence's last, from a zero state: its end state and the sum of its dt
//   chunk_pass    per state entry, over the chunks of a sequence: the chunks' start states
//   walk          every chunk from its start state, with the outputs
// (two exponentials per entry instead of one); else the walk starts from the request's state.  The float storage
// type walks in double, unchunked.  One token per sequence (decode): selective_step, which also makes the channel's
// raw step size from the low-rank row, raw_c = W_dt[c] . low[:R].
#include "common.cuh"
#include <type_traits>

namespace pmm {

constexpr int kSelThreads = 128;
constexpr int kSelTile = 16;  // tokens per shared-memory tile

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
// NPT neighbouring floats of shared memory (16-byte aligned where NPT is a multiple of 4).
template <int NPT>
__device__ __forceinline__ void sel_ld_shared(const float* p, float* o) {
  if (NPT % 4 == 0) {
#pragma unroll
    for (int i = 0; i < NPT; i += 4) {
      const float4 v = *reinterpret_cast<const float4*>(p + i);
      o[i] = v.x; o[i + 1] = v.y; o[i + 2] = v.z; o[i + 3] = v.w;
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < NPT; ++i) o[i] = p[i];
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

// OUT: the walk with outputs.  Otherwise chunk_state.
template <typename S, typename ACC, int LN, int NPT, bool OUT>
__global__ void __launch_bounds__(kSelThreads) selective_walk_kernel(const SelArgs p) {
  constexpr int CH = kSelThreads / LN;
  constexpr int NS = NPT + (NPT % 4 == 0 ? 4 : 0);  // a lane's entries of B or C (padded against bank conflicts)
  __shared__ ACC s_dt[kSelTile][CH], s_u[kSelTile][CH];
  __shared__ __align__(16) float s_b[kSelTile][LN * NS];
  __shared__ __align__(16) float s_c[OUT ? kSelTile : 1][LN * NS];
  __shared__ ACC s_y[OUT ? kSelTile : 1][CH + 1];
  pdl_launch_dependents();
  const int ch = threadIdx.x / LN, q = threadIdx.x % LN;
  const int c0 = blockIdx.x * CH, c = c0 + ch;
  const int N = p.N, I = p.I;
  const bool ch_ok = c < I;
  // constants of the channel: weights, read before the wait
  ACC a2[NPT];
#pragma unroll
  for (int i = 0; i < NPT; ++i) {
    const int n = q * NPT + i;
    a2[i] = (ch_ok && n < N) ? static_cast<ACC>(-1.4426950408889634) * scan_exp(static_cast<ACC>(p.a_log[static_cast<size_t>(c) * N + n])) : static_cast<ACC>(0);
  }
  pdl_wait();
  int seq, k, n_chunks;
  if (!sel_find_chunk(p.cu, p.n_seq, p.chunk_len, blockIdx.y, &seq, &k, &n_chunks)) return;
  if (!OUT && k == n_chunks - 1) return;  // nobody starts from a sequence's last chunk
  const int t_end = p.cu[seq + 1];
  const int t0 = p.cu[seq] + k * p.chunk_len, t1 = min(t_end, t0 + p.chunk_len);
  float* slot_state = p.state + (static_cast<size_t>(p.slots[seq]) * I + (ch_ok ? c : 0)) * N;
  float* mine = n_chunks > 1 ? p.chunk_state + (static_cast<size_t>(blockIdx.y) * I + (ch_ok ? c : 0)) * N : slot_state;
  const bool svec = N % 4 == 0;
  ACC st[NPT];
  {
    float f[NPT];
    if (OUT) sel_ld_state<NPT>(mine, q * NPT, N, svec, f);
#pragma unroll
    for (int i = 0; i < NPT; ++i) st[i] = OUT ? static_cast<ACC>(f[i]) : static_cast<ACC>(0);
  }
  ACC dt_sum = 0;

  // A tile's raw values wait in registers while the tile before it is walked.
  constexpr int PX = kSelTile * CH / kSelThreads;                     // (token, channel) pairs per thread
  constexpr int PB = (kSelTile * LN * NPT + kSelThreads - 1) / kSelThreads;  // (token, entry) pairs per thread
  float rx[PX], rd[PX], rz[OUT ? PX : 1], rb[PB], rc[OUT ? PB : 1];
  const S* xs = static_cast<const S*>(p.x);
  const S* ds = static_cast<const S*>(p.raw);
  const S* zs = static_cast<const S*>(p.z);
  const S* ls = static_cast<const S*>(p.low);
  auto request = [&](int base) {
#pragma unroll
    for (int r = 0; r < PX; ++r) {
      const int e = r * kSelThreads + threadIdx.x, tt = e / CH, cc = c0 + e % CH;
      const long long t = base + tt;
      const bool ok = t < t1 && cc < I;
      rx[r] = ok ? ldf(xs + t * p.ld_x + cc) : 0.f;
      rd[r] = ok ? ldf(ds + t * p.ld_raw + cc) : 0.f;
      if (OUT) rz[OUT ? r : 0] = ok ? ldf(zs + t * p.ld_z + cc) : 0.f;
    }
#pragma unroll
    for (int r = 0; r < PB; ++r) {
      const int e = r * kSelThreads + threadIdx.x, tt = e / (LN * NPT), n = e % (LN * NPT);
      const long long t = base + tt;
      const bool ok = tt < kSelTile && t < t1 && n < N;
      rb[r] = ok ? ldf(ls + t * p.ld_low + p.off_b + n) : 0.f;
      if (OUT) rc[OUT ? r : 0] = ok ? ldf(ls + t * p.ld_low + p.off_c + n) : 0.f;
    }
  };
  float bias[PX];
#pragma unroll
  for (int r = 0; r < PX; ++r) {
    const int cc = c0 + (r * kSelThreads + threadIdx.x) % CH;
    bias[r] = cc < I ? p.bias[cc] : 0.f;
  }
  request(t0);
  for (int base = t0; base < t1; base += kSelTile) {
    float zg[OUT ? PX : 1], xg[OUT ? PX : 1];
#pragma unroll
    for (int r = 0; r < PX; ++r) {
      const int e = r * kSelThreads + threadIdx.x, tt = e / CH, cc = e % CH;
      // (tokens past the chunk's end: dt = 0 leaves the state as it is)
      const ACC dt = base + tt < t1 ? scan_softplus<ACC>(static_cast<ACC>(rd[r]) + static_cast<ACC>(bias[r])) : static_cast<ACC>(0);
      s_dt[tt][cc] = dt;
      s_u[tt][cc] = dt * static_cast<ACC>(rx[r]);
      if (OUT) {
        xg[OUT ? r : 0] = rx[r];
        zg[OUT ? r : 0] = rz[OUT ? r : 0];
      }
    }
#pragma unroll
    for (int r = 0; r < PB; ++r) {
      const int e = r * kSelThreads + threadIdx.x, tt = e / (LN * NPT), n = e % (LN * NPT);
      if (tt < kSelTile) {
        s_b[tt][(n / NPT) * NS + n % NPT] = rb[r];
        if (OUT) s_c[OUT ? tt : 0][(n / NPT) * NS + n % NPT] = rc[OUT ? r : 0];
      }
    }
    __syncthreads();
    if (base + kSelTile < t1) request(base + kSelTile);
#pragma unroll 4
    for (int tt = 0; tt < kSelTile; ++tt) {
      const ACC dt = s_dt[tt][ch], u = s_u[tt][ch];
      ACC acc = 0;
      float bv[NPT], cv[NPT];
      sel_ld_shared<NPT>(&s_b[tt][q * NS], bv);
      if (OUT) sel_ld_shared<NPT>(&s_c[OUT ? tt : 0][q * NS], cv);
#pragma unroll
      for (int i = 0; i < NPT; ++i) {
        st[i] = sel_exp2(dt * a2[i]) * st[i] + u * static_cast<ACC>(bv[i]);
        if (OUT) acc += st[i] * static_cast<ACC>(cv[i]);
      }
      if (OUT) {
#pragma unroll
        for (int o = LN / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (q == 0) s_y[OUT ? tt : 0][ch] = acc;
      } else if (q == 0) {
        dt_sum += dt;
      }
    }
    __syncthreads();
    if (OUT) {
#pragma unroll
      for (int r = 0; r < PX; ++r) {
        const int e = r * kSelThreads + threadIdx.x, tt = e / CH, cc = c0 + e % CH;
        if (base + tt < t1 && cc < I) {
          const ACC y = s_y[tt][e % CH] + static_cast<ACC>(p.d[cc]) * static_cast<ACC>(xg[OUT ? r : 0]);
          const float g = sizeof(S) == 2 ? silu_fast(zg[OUT ? r : 0]) : silu_f(zg[OUT ? r : 0]);
          stf(static_cast<S*>(p.y) + static_cast<size_t>(base + tt) * I + cc, static_cast<float>(y) * g);
        }
      }
    }
  }
  if (!ch_ok) return;
  float* dst = OUT ? slot_state : mine;
  if (!OUT || k == n_chunks - 1) {
    float f[NPT];
#pragma unroll
    for (int i = 0; i < NPT; ++i) f[i] = static_cast<float>(st[i]);
    sel_st_state<NPT>(dst, q * NPT, N, svec, f);
  }
  if (!OUT && q == 0) p.chunk_dt[static_cast<size_t>(blockIdx.y) * I + c] = static_cast<float>(dt_sum);
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
__device__ __forceinline__ void sel_ld8(const float* p, float* o) {
#pragma unroll
  for (int i = 0; i < 8; ++i) o[i] = p[i];
}

// One token per sequence: token s of sequence s.  vec: rows of low and W_dt in whole pieces of 8 elements.
template <typename S, typename ACC, int LN, int NPT>
__global__ void __launch_bounds__(kSelThreads) selective_step_kernel(const SelArgs p, int vec) {
  constexpr int CH = kSelThreads / LN;
  pdl_launch_dependents();
  const int ch = threadIdx.x / LN, q = threadIdx.x % LN;
  const int c = blockIdx.x * CH + ch;
  const int s = blockIdx.y;
  const int N = p.N, I = p.I;
  const bool ok = c < I;
  const int cs = ok ? c : 0;
  ACC a2[NPT];
#pragma unroll
  for (int i = 0; i < NPT; ++i) {
    const int n = q * NPT + i;
    a2[i] = (ok && n < N) ? static_cast<ACC>(-1.4426950408889634) * scan_exp(static_cast<ACC>(p.a_log[static_cast<size_t>(cs) * N + n])) : static_cast<ACC>(0);
  }
  const ACC bias = p.bias[cs], dskip = p.d[cs];
  const int slot = p.slots[s];
  pdl_wait();
  float* srow = p.state + (static_cast<size_t>(slot) * I + cs) * N;
  const bool svec = N % 4 == 0;
  float st[NPT];
  sel_ld_state<NPT>(srow, q * NPT, N, svec, st);
  const S* low = static_cast<const S*>(p.low) + static_cast<long long>(s) * p.ld_low;
  const S* w = static_cast<const S*>(p.w_dt) + static_cast<size_t>(cs) * p.R;
  ACC raw = 0;
  if (vec) {
    for (int r = q * 8; r < p.R; r += LN * 8) {
      float lv[8], wv[8];
      sel_ld8(low + r, lv);
      sel_ld8(w + r, wv);
#pragma unroll
      for (int i = 0; i < 8; ++i) raw += static_cast<ACC>(lv[i]) * static_cast<ACC>(wv[i]);
    }
  } else {
    for (int r = q; r < p.R; r += LN) raw += static_cast<ACC>(ldf(low + r)) * static_cast<ACC>(ldf(w + r));
  }
#pragma unroll
  for (int o = LN / 2; o > 0; o >>= 1) raw += __shfl_xor_sync(0xffffffffu, raw, o);
  const ACC dt = scan_softplus<ACC>(raw + bias);
  const ACC xv = ldf(static_cast<const S*>(p.x) + static_cast<long long>(s) * p.ld_x + cs);
  const ACC u = dt * xv;
  ACC acc = 0;
#pragma unroll
  for (int i = 0; i < NPT; ++i) {
    const int n = q * NPT + i;
    if (ok && n < N) {
      const ACC v = sel_exp2(dt * a2[i]) * static_cast<ACC>(st[i]) + u * static_cast<ACC>(ldf(low + p.off_b + n));
      acc += v * static_cast<ACC>(ldf(low + p.off_c + n));
      st[i] = static_cast<float>(v);
    }
  }
  if (ok) sel_st_state<NPT>(srow, q * NPT, N, svec, st);
#pragma unroll
  for (int o = LN / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
  if (ok && q == 0) {
    const float zv = ldf(static_cast<const S*>(p.z) + static_cast<long long>(s) * p.ld_z + c);
    stf(static_cast<S*>(p.y) + static_cast<size_t>(s) * I + c, static_cast<float>(acc + dskip * xv) * silu_f(zv));
  }
}

// Lanes per channel and entries per lane for N state entries.
#define PMM_SEL_DISPATCH(N, CALL)      \
  do {                                 \
    if ((N) <= 4) { CALL(4, 1); }      \
    else if ((N) <= 8) { CALL(4, 2); } \
    else if ((N) <= 12) { CALL(4, 3); } \
    else if ((N) <= 16) { CALL(4, 4); } \
    else if ((N) <= 24) { CALL(8, 3); } \
    else if ((N) <= 32) { CALL(8, 4); } \
    else if ((N) <= 48) { CALL(16, 3); } \
    else if ((N) <= 64) { CALL(16, 4); } \
    else if ((N) <= 128) { CALL(16, 8); } \
    else { CALL(16, 16); }             \
  } while (0)

inline int sel_lanes(int N) { return N <= 16 ? 4 : N <= 32 ? 8 : 16; }

template <typename S, bool OUT>
int launch_selective_walk(const SelArgs& p, int n_chunks, cudaStream_t stream) {
  using ACC = typename std::conditional<sizeof(S) == 4, double, float>::type;
  const int ch = kSelThreads / sel_lanes(p.N);
  dim3 grid((p.I + ch - 1) / ch, n_chunks);
#define PMM_SEL_WALK(LN, NPT) launch_pdl(selective_walk_kernel<S, ACC, LN, NPT, OUT>, grid, dim3(kSelThreads), 0, stream, p)
  PMM_SEL_DISPATCH(p.N, PMM_SEL_WALK);
#undef PMM_SEL_WALK
  return launch_status();
}

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
PMM_EXPORT int pmm_selective_scan_channels(int N) { return N <= 0 || N > 256 ? 0 : pmm::kSelThreads / pmm::sel_lanes(N); }

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
                 slots, y, n_seq, I, N, chunk_len, nullptr, 0};
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
// w_dt [I, R] contiguous.
PMM_EXPORT int pmm_selective_step(const void* x, long long ld_x, const void* low, long long ld_low, int R, int off_b, int off_c,
                                  const void* w_dt, const void* z, long long ld_z, const float* bias, const float* a_log,
                                  const float* d, float* state, const int* slots, void* y, int n_seq, int I, int N, int dtype,
                                  cudaStream_t stream) {
  if (n_seq <= 0) return 0;
  if (I <= 0 || N <= 0 || N > 256 || R <= 0 || n_seq > 65535) return PMM_ERR_BAD_ARGUMENT;
  pmm::SelArgs p{x, nullptr, low, z, ld_x, 0, ld_low, ld_z, off_b, off_c, bias, a_log, d, state, nullptr, nullptr, nullptr,
                 slots, y, n_seq, I, N, 0, w_dt, R};
  const int vec = R % 8 == 0 && ld_low % 8 == 0 && reinterpret_cast<uintptr_t>(low) % 16 == 0 && reinterpret_cast<uintptr_t>(w_dt) % 16 == 0;
  PMM_DISPATCH_DTYPE(dtype, S, return pmm::launch_selective_step<S>(p, vec, stream));
  return 0;
}
