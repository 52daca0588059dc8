// The residual fold with an RMS norm over groups of channels and, where the sublayer has one, the causal
// convolution of its input, in one launch:
//
//   v_t   = h_t + sa * a_t + sb * b_t + vec            (the waiting branches and a vector join the stream)
//   n_t,c = v_t,c / sqrt(mean over c's group of v_t^2 + eps) * w_c
//   y_t   = n_t + sum_j k[j, c] * n_(t - L + j),  j = 0 .. L,  L = taps - 1      (with a convolution)
//
// The stream, the statistics, the normed rows and the convolution are float; a, b and y have the storage type.
// Inputs before a portion come from the request's window [slot][L][D] (float, oldest first, zero for a new
// request), which the launch leaves holding the last L normed rows of every sequence.
//
// The convolution needs the normed rows of the L tokens before each token.  They are not kept: a block takes a
// tile of rows, computes the statistics of its rows and of the L rows before them, and walks them column by
// column with the last L normed values in registers.  Other blocks read the same rows of h, so the folded stream
// goes to a second buffer (h_out != h_in) unless every sequence brings one token.  What touches a window is left to
// one block per sequence ("head" block): it makes the outputs of the sequence's first L tokens, which are the
// only ones that read the window, and then writes the new window; a tile block leaves those tokens' outputs alone.
// No other block reads or writes that window, so one launch serves portions of any length.
#include "common.cuh"

namespace pmm {

constexpr int kFoldMaxWarps = 16;

struct FoldArgs {
  const float* h_in;
  float* h_out;         // may be h_in when no row is read by two blocks
  const void* a;
  const void* b;
  float sa, sb;
  const float* vec;     // [D] or nullptr
  const float* w;       // [D], nullptr: fold only
  float eps;
  int groups;
  const float* conv;    // [taps][D] (tap-major) or nullptr
  int taps;
  float* window;
  const int* cu;
  const int* slots;
  const int* seq_of;
  const int* rows;      // chosen rows (no fold into h, no convolution) or nullptr
  void* out;
  int T, D;
  int n_tiles, tile_rows;  // tile blocks come first in the grid, then one head block per sequence
  int fold_in_heads;       // the head blocks write h_out (every sequence brings one token, there are no tiles)
};

template <int V>
struct Cols {
  float v[V];
};

__device__ __forceinline__ void fold_ld(const float* p, Cols<4>& o) {
  const float4 x = *reinterpret_cast<const float4*>(p);
  o.v[0] = x.x; o.v[1] = x.y; o.v[2] = x.z; o.v[3] = x.w;
}
__device__ __forceinline__ void fold_ld(const __nv_bfloat16* p, Cols<4>& o) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  o.v[0] = x.x; o.v[1] = x.y; o.v[2] = y.x; o.v[3] = y.y;
}
template <typename S>
__device__ __forceinline__ void fold_ld(const S* p, Cols<1>& o) { o.v[0] = ldf(p); }
__device__ __forceinline__ void fold_st(float* p, const Cols<4>& o) {
  *reinterpret_cast<float4*>(p) = make_float4(o.v[0], o.v[1], o.v[2], o.v[3]);
}
__device__ __forceinline__ void fold_st(__nv_bfloat16* p, const Cols<4>& o) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(o.v[0], o.v[1]);
  *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(o.v[2], o.v[3]);
  *reinterpret_cast<uint2*>(p) = raw;
}
template <typename S>
__device__ __forceinline__ void fold_st(S* p, const Cols<1>& o) { stf(p, o.v[0]); }

// Row `row` of the folded stream, columns c .. c + V - 1.
template <typename S, int V>
__device__ __forceinline__ Cols<V> folded(const FoldArgs& p, int row, int c) {
  const size_t at = static_cast<size_t>(row) * p.D + c;
  Cols<V> v, x;
  fold_ld(p.h_in + at, v);
  if (p.a) {
    fold_ld(static_cast<const S*>(p.a) + at, x);
#pragma unroll
    for (int i = 0; i < V; ++i) v.v[i] += p.sa * x.v[i];
  }
  if (p.b) {
    fold_ld(static_cast<const S*>(p.b) + at, x);
#pragma unroll
    for (int i = 0; i < V; ++i) v.v[i] += p.sb * x.v[i];
  }
  if (p.vec) {
    fold_ld(p.vec + c, x);
#pragma unroll
    for (int i = 0; i < V; ++i) v.v[i] += x.v[i];
  }
  return v;
}

// LR: taps - 1 where the history fits registers (0 .. 3), -1: any number of taps, history in shared memory.
template <typename S, int LR, int V>
__global__ void __launch_bounds__(kFoldMaxWarps * 32) fold_norm_kernel(const FoldArgs p) {
  extern __shared__ float fold_smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int L = LR >= 0 ? LR : p.taps - 1;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  const bool head = static_cast<int>(blockIdx.x) >= p.n_tiles;

  // The block's list of rows: list index i is token first + i, from `gap` on shifted by `skip` (a head block of a
  // long portion takes its first L and its last L rows).
  int first, count, gap = 0x7fffffff, skip = 0, own = 0, slot = 0, seq_first = 0;
  if (!head) {
    const int t0 = blockIdx.x * p.tile_rows;
    first = max(t0 - L, 0);
    own = t0 - first;                                  // list indices from here on are the tile's own rows
    count = own + min(p.tile_rows, p.T - t0);
  } else {
    const int s = blockIdx.x - p.n_tiles;
    seq_first = p.cu[s];
    const int n = p.cu[s + 1] - seq_first;
    if (n <= 0) return;
    slot = p.slots[s];
    first = seq_first;
    count = min(n, 2 * L);
    if (n > 2 * L) { gap = L; skip = n - 2 * L; }
  }
  auto token = [&](int i) { return p.rows ? p.rows[first + i] : first + i + (i >= gap ? skip : 0); };

  // statistics: inv[list index][group]; several warps share a row where there are more warps than rows
  float* inv = fold_smem;
  const int groups = p.groups, gw = p.D / groups;
  if (p.w) {
    int wpr = n_warps / count;
    if (wpr < 1) wpr = 1;
    float* part = inv + static_cast<size_t>(max(p.tile_rows + L, 2 * L)) * groups;  // [row in round][group][wpr]
    const int per_round = n_warps / wpr;
    const int my_row = warp / wpr, my_part = warp % wpr;
    for (int base = 0; base < count; base += per_round) {
      const int i = base + my_row;
      if (my_row < per_round && i < count) {
        const int row = token(i);
        for (int g = 0; g < groups; ++g) {
          float ss = 0.f;
#pragma unroll 4
          for (int c = (my_part * 32 + lane) * V; c < gw; c += wpr * 32 * V) {
            const Cols<V> v = folded<S, V>(p, row, g * gw + c);
#pragma unroll
            for (int e = 0; e < V; ++e) ss += v.v[e] * v.v[e];
          }
          ss = warp_sum(ss);
          if (lane == 0) part[(my_row * groups + g) * wpr + my_part] = ss;
        }
      }
      __syncthreads();
      for (int k = threadIdx.x; k < per_round * groups; k += blockDim.x) {
        const int r = k / groups, g = k - r * groups;
        if (base + r < count) {
          float ss = 0.f;
          for (int q = 0; q < wpr; ++q) ss += part[k * wpr + q];
          inv[(base + r) * groups + g] = 1.f / sqrtf(ss / static_cast<float>(gw) + p.eps);
        }
      }
      __syncthreads();
    }
  }

  constexpr int H = LR > 0 ? LR : 1;
  // LR < 0: history [L][threads * V], on a 16-byte boundary
  float* far = fold_smem + (((static_cast<size_t>(max(p.tile_rows + L, 2 * L)) + kFoldMaxWarps) * groups + 3) & ~static_cast<size_t>(3));
  const bool fold = !p.rows && (head ? p.fold_in_heads != 0 : true) && (p.a || p.b || p.vec || p.h_out != p.h_in);
  for (int c = threadIdx.x * V; c < p.D; c += blockDim.x * V) {
    Cols<V> w, kt[H + 1], hist[H];
    if (p.w) fold_ld(p.w + c, w);
    if (p.conv && LR >= 0) {
#pragma unroll
      for (int j = 0; j <= (LR > 0 ? LR : 0); ++j) fold_ld(p.conv + static_cast<size_t>(j) * p.D + c, kt[j]);
    }
    const int g = c / gw;
    auto far_at = [&](int k) { return far + (static_cast<size_t>(k % L) * blockDim.x + threadIdx.x) * V; };
    if (head) {  // the last L inputs before the portion
      const float* win = p.window + static_cast<size_t>(slot) * L * p.D + c;
      if (LR > 0) {
#pragma unroll
        for (int k = 0; k < LR; ++k) fold_ld(win + static_cast<size_t>(k) * p.D, hist[k]);
      } else if (LR < 0) {
        for (int k = 0; k < L; ++k) {
          Cols<V> x;
          fold_ld(win + static_cast<size_t>(k) * p.D, x);
          fold_st(far_at(k), x);
        }
      }
    } else if (LR > 0) {
#pragma unroll
      for (int k = 0; k < LR; ++k)
#pragma unroll
        for (int e = 0; e < V; ++e) hist[k].v[e] = 0.f;
    }
    constexpr int B = 4;  // rows requested together
    for (int base = 0; base < count; base += B) {
      Cols<V> v[B];
#pragma unroll
      for (int q = 0; q < B; ++q)
        if (base + q < count) v[q] = folded<S, V>(p, token(base + q), c);
#pragma unroll
      for (int q = 0; q < B; ++q) {
        const int i = base + q;
        if (i >= count) break;
        const int t = token(i);
        if (fold && (head || i >= own)) fold_st(p.h_out + static_cast<size_t>(t) * p.D + c, v[q]);
        if (!p.w) continue;
        const float scale = inv[i * groups + g];
        Cols<V> n, y;
#pragma unroll
        for (int e = 0; e < V; ++e) n.v[e] = v[q].v[e] * scale * w.v[e];
        // whose output is it: a head block writes the sequence's first L tokens, a tile block the others
        const int j = (head || L == 0 || !p.conv) ? 0 : t - p.cu[p.seq_of[t]];
        const bool mine = head ? t - seq_first < L : (i >= own && j >= L) || !p.conv;
        if (p.conv && LR >= 0) {
#pragma unroll
          for (int e = 0; e < V; ++e) {
            float acc = 0.f;
#pragma unroll
            for (int k = 0; k < (LR > 0 ? LR : 0); ++k) acc += kt[k].v[e] * hist[k].v[e];
            acc += kt[LR > 0 ? LR : 0].v[e] * n.v[e];
            y.v[e] = n.v[e] + acc;
          }
        } else if (p.conv) {
          // list index i: history entry k (0 = oldest) of the last L inputs sits at ring place i + k
          Cols<V> kc;
#pragma unroll
          for (int e = 0; e < V; ++e) y.v[e] = 0.f;
          if (mine) {
            for (int k = 0; k < L; ++k) {
              Cols<V> x;
              fold_ld(far_at(i + k), x);
              fold_ld(p.conv + static_cast<size_t>(k) * p.D + c, kc);
#pragma unroll
              for (int e = 0; e < V; ++e) y.v[e] += kc.v[e] * x.v[e];
            }
            fold_ld(p.conv + static_cast<size_t>(L) * p.D + c, kc);
#pragma unroll
            for (int e = 0; e < V; ++e) y.v[e] = n.v[e] + (y.v[e] + kc.v[e] * n.v[e]);
          }
          fold_st(far_at(i), n);  // replaces the oldest
        } else {
          y = n;
        }
        if (LR > 0) {
#pragma unroll
          for (int k = 0; k + 1 < LR; ++k) hist[k] = hist[k + 1];
          hist[H - 1] = n;
        }
        if (mine) fold_st(static_cast<S*>(p.out) + static_cast<size_t>(p.rows ? first + i : t) * p.D + c, y);
      }
    }
    if (head) {
      float* win = p.window + static_cast<size_t>(slot) * L * p.D + c;
      if (LR > 0) {
#pragma unroll
        for (int k = 0; k < LR; ++k) fold_st(win + static_cast<size_t>(k) * p.D, hist[k]);
      } else if (LR < 0) {
        for (int k = 0; k < L; ++k) {
          Cols<V> x;
          fold_ld(far_at(count + k), x);
          fold_st(win + static_cast<size_t>(k) * p.D, x);
        }
      }
    }
  }
}

template <typename S, int LR, int V>
int launch_fold_norm(const FoldArgs& p, int n_heads, int threads, size_t smem, cudaStream_t stream) {
  auto kern = fold_norm_kernel<S, LR, V>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  launch_pdl(kern, dim3(p.n_tiles + n_heads), dim3(threads), smem, stream, p);
  return launch_status();
}

template <typename S, int V>
int dispatch_fold_norm(const FoldArgs& p, int n_heads, int threads, size_t smem, cudaStream_t stream) {
  switch (p.conv ? p.taps - 1 : 0) {
    case 0: return launch_fold_norm<S, 0, V>(p, n_heads, threads, smem, stream);
    case 1: return launch_fold_norm<S, 1, V>(p, n_heads, threads, smem, stream);
    case 2: return launch_fold_norm<S, 2, V>(p, n_heads, threads, smem, stream);
    case 3: return launch_fold_norm<S, 3, V>(p, n_heads, threads, smem, stream);
    default: return launch_fold_norm<S, -1, V>(p, n_heads, threads, smem, stream);
  }
}

}  // namespace pmm

// h_in, h_out [T, D] float; a, b [T, D] storage type or nullptr; vec [D] float or nullptr; w [D] float (nullptr: fold
// only, out nullptr as well); conv [taps][D] float or nullptr; window [slots, taps - 1, D] float (taps > 1); cu, slots,
// seq_of: with a convolution; rows [R] or nullptr: the norm of those rows only, h as it is (R == T then counts them).
// one_token: every sequence brings exactly one token.  out [T (R), D] storage type.
PMM_EXPORT int pmm_fold_norm(const float* h_in, float* h_out, const void* a, float sa, const void* b, float sb,
                             const float* vec, const float* w, float eps, int groups, const float* conv, int taps,
                             float* window, const int* cu, const int* slots, const int* seq_of, int n_seq, int one_token,
                             const int* rows, void* out, int T, int D, int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (D <= 0 || groups <= 0 || D % groups || !h_in || (w && !out) || (!w && (conv || rows)) || (conv && rows)) return PMM_ERR_BAD_ARGUMENT;
  if (conv && (taps < 1 || (taps > 1 && (!window || !cu || !slots || !seq_of || n_seq <= 0)))) return PMM_ERR_BAD_ARGUMENT;
  const int L = conv ? taps - 1 : 0;
  if (!rows && !h_out) return PMM_ERR_BAD_ARGUMENT;
  // rows that two blocks read must not be written in place
  if (L > 0 && !one_token && h_out == h_in && (a || b || vec)) return PMM_ERR_BAD_ARGUMENT;
  auto aligned = [](const void* q) { return reinterpret_cast<uintptr_t>(q) % 16 == 0; };
  const bool vec4 = (D / groups) % 4 == 0 && aligned(h_in) && aligned(h_out) && aligned(a) && aligned(b) && aligned(vec) && aligned(w) &&
                    aligned(conv) && aligned(window) && aligned(out);
  const int V = vec4 ? 4 : 1;
  int warps = (D / V + 31) / 32;
  if (warps < 4) warps = 4;
  if (warps > pmm::kFoldMaxWarps) warps = pmm::kFoldMaxWarps;
  const bool heads_only = L > 0 && one_token;
  pmm::FoldArgs p{h_in, h_out, a, b, sa, sb, vec, w, eps, groups, conv, taps, window, cu, slots, seq_of, rows, out, T, D,
                  0, 1, heads_only ? 1 : 0};
  // with a convolution a tile has as many rows (its own and the L before them) as the block has warps
  if (L > 0) p.tile_rows = warps > L + 1 ? warps - L : (L < 8 ? 8 : L);
  p.n_tiles = heads_only ? 0 : (T + p.tile_rows - 1) / p.tile_rows;
  const int n_heads = L > 0 ? n_seq : 0;
  const int threads = warps * 32;
  const int list = p.tile_rows + L > 2 * L ? p.tile_rows + L : 2 * L;
  size_t smem = (static_cast<size_t>(list) * groups + static_cast<size_t>(pmm::kFoldMaxWarps) * groups) * sizeof(float);
  if (L > 3) smem = (smem + 15) / 16 * 16 + static_cast<size_t>(L) * threads * V * sizeof(float);
  if (smem > 200 * 1024) return PMM_ERR_BAD_ARGUMENT;
  PMM_DISPATCH_DTYPE(dtype, S, {
    if (vec4) return pmm::dispatch_fold_norm<S, 4>(p, n_heads, threads, smem, stream);
    return pmm::dispatch_fold_norm<S, 1>(p, n_heads, threads, smem, stream);
  });
  return 0;
}
