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
//
// Rows that nobody else reads (no convolution, one tap, or one token per sequence) take fold_norm_row: a block per row,
// the row in registers from its one read to its one write, constants and the window requested before the reduction.
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
  int far_at;              // where in shared memory the history of many taps begins (floats)
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

// How a row's squares are summed by group.  A piece is 32 lanes x 4 columns = 128 columns.
//   kGroupWarp: a group is a whole number of pieces: every piece leaves one sum, a group adds up its pieces
//   kGroupLanes: a group is 1, 2, 4, .. 16 lanes of a piece: shuffles within those lanes
//   kGroupAny: anything else: group by group
enum { kGroupWarp = 0, kGroupLanes = 1, kGroupAny = 2 };

__device__ __forceinline__ float lanes_sum(float v, int lanes) {  // sum over aligned runs of `lanes` (a power of two) lanes
  for (int o = lanes >> 1; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// A block per row (see the top of the file).  P pieces of 4 columns per thread; groups: kGroupWarp or kGroupLanes.
template <typename S, int LR, int P>
__global__ void __launch_bounds__(kFoldMaxWarps * 32) fold_norm_row_kernel(const FoldArgs p, int mode) {
  __shared__ float part[kFoldMaxWarps * P];
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  const int D = p.D, gw = D / p.groups;
  const int step = blockDim.x * 4;
  constexpr int H = LR > 0 ? LR : 1;
  Cols<4> v[P], w[P], hist[P][H];
#pragma unroll
  for (int c = 0; c < P; ++c) {  // constants: weights, read before the wait
    const int i = threadIdx.x * 4 + c * step;
    if (p.w && i < D) fold_ld(p.w + i, w[c]);
  }
  pdl_wait();
  const int r = blockIdx.x;
  const int t = p.rows ? p.rows[r] : r;
  const float* win = nullptr;
  if (LR > 0) win = p.window + static_cast<size_t>(p.slots[r]) * LR * D;
#pragma unroll
  for (int c = 0; c < P; ++c) {
    const int i = threadIdx.x * 4 + c * step;
    if (i < D) {
      v[c] = folded<S, 4>(p, t, i);
    } else {
      v[c].v[0] = v[c].v[1] = v[c].v[2] = v[c].v[3] = 0.f;
    }
  }
  if (LR > 0) {
#pragma unroll
    for (int c = 0; c < P; ++c) {
      const int i = threadIdx.x * 4 + c * step;
      if (i < D) {
#pragma unroll
        for (int k = 0; k < LR; ++k) fold_ld(win + static_cast<size_t>(k) * D + i, hist[c][k]);
      }
    }
  }
  if (!p.rows && (p.a || p.b || p.vec || p.h_out != p.h_in)) {
#pragma unroll
    for (int c = 0; c < P; ++c) {
      const int i = threadIdx.x * 4 + c * step;
      if (i < D) fold_st(p.h_out + static_cast<size_t>(t) * D + i, v[c]);
    }
  }
  if (!p.w) return;
  float scale[P];
  if (mode == kGroupWarp) {
#pragma unroll
    for (int c = 0; c < P; ++c) {
      const float ss = warp_sum(v[c].v[0] * v[c].v[0] + v[c].v[1] * v[c].v[1] + v[c].v[2] * v[c].v[2] + v[c].v[3] * v[c].v[3]);
      if (lane == 0) part[c * n_warps + warp] = ss;  // piece number: c * n_warps + warp
    }
    __syncthreads();
    const int per = gw / 128;  // pieces of a group
#pragma unroll
    for (int c = 0; c < P; ++c) {
      const int first = (c * n_warps + warp) / per * per;
      float ss = 0.f;
      for (int k = lane; k < per; k += 32) ss += first + k < P * n_warps ? part[first + k] : 0.f;
      scale[c] = rsqrtf(warp_sum(ss) / static_cast<float>(gw) + p.eps);
    }
  } else {
#pragma unroll
    for (int c = 0; c < P; ++c) {
      const float ss = lanes_sum(v[c].v[0] * v[c].v[0] + v[c].v[1] * v[c].v[1] + v[c].v[2] * v[c].v[2] + v[c].v[3] * v[c].v[3], gw / 4);
      scale[c] = rsqrtf(ss / static_cast<float>(gw) + p.eps);
    }
  }
#pragma unroll
  for (int c = 0; c < P; ++c) {
    const int i = threadIdx.x * 4 + c * step;
    if (i >= D) continue;
    Cols<4> n, y;
#pragma unroll
    for (int e = 0; e < 4; ++e) n.v[e] = v[c].v[e] * scale[c] * w[c].v[e];
    y = n;
    if (p.conv) {
      Cols<4> kt, acc;
#pragma unroll
      for (int e = 0; e < 4; ++e) acc.v[e] = 0.f;
#pragma unroll
      for (int k = 0; k <= (LR > 0 ? LR : 0); ++k) {
        fold_ld(p.conv + static_cast<size_t>(k) * D + i, kt);
#pragma unroll
        for (int e = 0; e < 4; ++e) acc.v[e] += kt.v[e] * (k < (LR > 0 ? LR : 0) ? hist[c][k < H ? k : 0].v[e] : n.v[e]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) y.v[e] = n.v[e] + acc.v[e];
      if (LR > 0) {
        float* dst = p.window + static_cast<size_t>(p.slots[r]) * LR * D + i;
#pragma unroll
        for (int k = 0; k + 1 < LR; ++k) fold_st(dst + static_cast<size_t>(k) * D, hist[c][k + 1]);
        fold_st(dst + static_cast<size_t>(LR - 1) * D, n);
      }
    }
    fold_st(static_cast<S*>(p.out) + static_cast<size_t>(r) * D + i, y);
  }
}

// The rows of a strip one after the other, each read once (kGroupWarp or kGroupLanes, 2 to 4 taps): a thread owns P pieces
// of 4 columns, two rows are normed between two block barriers, and the last LR normed rows stay in registers.  The rows
// come by asynchronous copies into the thread's own places of a ring of kFoldWalkPairs pairs of rows, so that the pairs
// after the one at hand are on their way.  Tile and head blocks as in fold_norm_kernel.
constexpr int kFoldWalkPairs = 3;
constexpr int kFoldWalkRows = 64;  // rows of a strip, with the ones before it
template <int P>
struct FoldWalk {
  static constexpr int kThreads = P == 1 ? 768 : 512;
};

template <int BYTES>
__device__ __forceinline__ void fold_copy(void* dst, const void* src) {
  const unsigned d = static_cast<unsigned>(__cvta_generic_to_shared(dst));
  if (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(d), "l"(src) : "memory");
}

template <typename S, int LR, int P>
__global__ void __launch_bounds__(FoldWalk<P>::kThreads, 1) fold_norm_walk_kernel(const FoldArgs p, int mode) {
  extern __shared__ __align__(16) unsigned char fold_ring[];  // [pair][row of the pair][P]: floats of h (16 bytes a thread), then a
  __shared__ float part[2][2][FoldWalk<P>::kThreads / 32 * P * 2];  // (a group's pieces are read beyond the last one)
  __shared__ int place[kFoldWalkRows];
  constexpr int AB = 4 * sizeof(S);  // bytes of a thread's piece of a
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  const int D = p.D, gw = D / p.groups, step = blockDim.x * 4;
  const S* pa = static_cast<const S*>(p.a);
  Cols<4> w[P], kt[P][LR + 1], hist[P][LR];
#pragma unroll
  for (int c = 0; c < P; ++c) {  // constants: weights, read before the wait
    const int i = threadIdx.x * 4 + c * step;
    if (i < D) {
      fold_ld(p.w + i, w[c]);
#pragma unroll
      for (int k = 0; k <= LR; ++k) fold_ld(p.conv + static_cast<size_t>(k) * D + i, kt[c][k]);
    }
  }
  pdl_wait();
  const bool head = static_cast<int>(blockIdx.x) >= p.n_tiles;
  int first, count, gap = 0x7fffffff, skip = 0, own = 0;
  float* win = nullptr;
  if (!head) {
    const int t0 = blockIdx.x * p.tile_rows;
    first = max(t0 - LR, 0);
    own = t0 - first;
    count = own + min(p.tile_rows, p.T - t0);
  } else {
    const int s = blockIdx.x - p.n_tiles;
    first = p.cu[s];
    const int n = p.cu[s + 1] - first;
    if (n <= 0) return;
    count = min(n, 2 * LR);
    if (n > 2 * LR) { gap = LR; skip = n - 2 * LR; }
    win = p.window + static_cast<size_t>(p.slots[s]) * LR * D;
  }
  auto token = [&](int i) { return first + i + (i >= gap ? skip : 0); };
  auto h_at = [&](int slot, int q, int c) {
    return fold_ring + (static_cast<size_t>((slot * 2 + q) * P + c) * blockDim.x + threadIdx.x) * 16;
  };
  auto a_at = [&](int slot, int q, int c) {
    return fold_ring + static_cast<size_t>(kFoldWalkPairs * 2 * P) * blockDim.x * 16 +
           (static_cast<size_t>((slot * 2 + q) * P + c) * blockDim.x + threadIdx.x) * AB;
  };
  auto request = [&](int base, int slot) {
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      if (base + q < count) {
        const size_t row = static_cast<size_t>(token(base + q)) * D;
#pragma unroll
        for (int c = 0; c < P; ++c) {
          const int i = threadIdx.x * 4 + c * step;
          if (i < D) {
            fold_copy<16>(h_at(slot, q, c), p.h_in + row + i);
            if (pa) fold_copy<AB>(a_at(slot, q, c), pa + row + i);
          }
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int k = 0; k < kFoldWalkPairs - 1; ++k) request(2 * k, k);
  if (!head) {
    for (int i = threadIdx.x; i < count; i += blockDim.x) place[i] = first + i - p.cu[p.seq_of[first + i]];
    __syncthreads();
  }
#pragma unroll
  for (int c = 0; c < P; ++c) {
    const int i = threadIdx.x * 4 + c * step;
#pragma unroll
    for (int k = 0; k < LR; ++k) {
      if (head && i < D) {
        fold_ld(win + static_cast<size_t>(k) * D + i, hist[c][k]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) hist[c][k].v[e] = 0.f;
      }
    }
  }
  const int per = mode == kGroupWarp ? gw / 128 : 1;
  const float inv_gw = 1.f / static_cast<float>(gw);
  int group_at[P];  // the first piece of this thread's group
#pragma unroll
  for (int c = 0; c < P; ++c) group_at[c] = (c * n_warps + warp) / per * per;
  int slot = 0, buf = 0;
#pragma unroll 1
  for (int base = 0; base < count; base += 2) {
    request(base + 2 * (kFoldWalkPairs - 1), slot == 0 ? kFoldWalkPairs - 1 : slot - 1);  // (the pair before this one has left its place)
    asm volatile("cp.async.wait_group %0;" ::"n"(kFoldWalkPairs - 1) : "memory");
    Cols<4> v[2][P];
    float scale[2][P], ss[2][P];
#pragma unroll
    for (int q = 0; q < 2; ++q) {
#pragma unroll
      for (int c = 0; c < P; ++c) {
        const int i = threadIdx.x * 4 + c * step;
        ss[q][c] = 0.f;
        if (base + q < count && i < D) {
          fold_ld(reinterpret_cast<const float*>(h_at(slot, q, c)), v[q][c]);
          Cols<4> x;
          if (pa) {
            fold_ld(reinterpret_cast<const S*>(a_at(slot, q, c)), x);
#pragma unroll
            for (int e = 0; e < 4; ++e) v[q][c].v[e] += p.sa * x.v[e];
          }
          if (p.b) {
            fold_ld(static_cast<const S*>(p.b) + static_cast<size_t>(token(base + q)) * D + i, x);
#pragma unroll
            for (int e = 0; e < 4; ++e) v[q][c].v[e] += p.sb * x.v[e];
          }
          if (p.vec) {
            fold_ld(p.vec + i, x);
#pragma unroll
            for (int e = 0; e < 4; ++e) v[q][c].v[e] += x.v[e];
          }
#pragma unroll
          for (int e = 0; e < 4; ++e) ss[q][c] += v[q][c].v[e] * v[q][c].v[e];
        }
      }
    }
    if (mode == kGroupWarp) {
#pragma unroll
      for (int c = 0; c < P; ++c) {
        // both rows at once: the lower half of the warp sums the first, the upper half the second
        const bool up = lane >= 16;
        float sum = (up ? ss[1][c] : ss[0][c]) + __shfl_xor_sync(0xffffffffu, up ? ss[0][c] : ss[1][c], 16);
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        if ((lane & 15) == 0) part[buf][lane >> 4][c * n_warps + warp] = sum;
      }
      __syncthreads();  // (the other buffer takes the next pair, so one barrier a pair is enough)
#pragma unroll
      for (int q = 0; q < 2; ++q) {
#pragma unroll
        for (int c = 0; c < P; ++c) {
          const float* pieces = &part[buf][q][group_at[c]];
          float sum = 0.f;
          if (per <= 4) {
            for (int k = 0; k < per; ++k) sum += pieces[k];
          } else {
            for (int k = lane; k < per; k += 32) sum += pieces[k];
            sum = warp_sum(sum);
          }
          scale[q][c] = rsqrtf(sum * inv_gw + p.eps);
        }
      }
    } else {
#pragma unroll
      for (int q = 0; q < 2; ++q)
#pragma unroll
        for (int c = 0; c < P; ++c) scale[q][c] = rsqrtf(lanes_sum(ss[q][c], gw / 4) * inv_gw + p.eps);
    }
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int li = base + q;
      if (li < count) {
        const size_t row = static_cast<size_t>(token(li)) * D;
        const bool keep = !head && li >= own;               // the stream's row is this block's to write
        const bool mine = head ? li < LR : keep && place[li] >= LR;
#pragma unroll
        for (int c = 0; c < P; ++c) {
          const int i = threadIdx.x * 4 + c * step;
          if (i < D) {
            if (keep && p.h_out != p.h_in) fold_st(p.h_out + row + i, v[q][c]);
            Cols<4> n, y;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              n.v[e] = v[q][c].v[e] * scale[q][c] * w[c].v[e];
              float acc = 0.f;
#pragma unroll
              for (int k = 0; k < LR; ++k) acc += kt[c][k].v[e] * hist[c][k].v[e];
              acc += kt[c][LR].v[e] * n.v[e];
              y.v[e] = n.v[e] + acc;
            }
#pragma unroll
            for (int k = 0; k + 1 < LR; ++k) hist[c][k] = hist[c][k + 1];
            hist[c][LR - 1] = n;
            if (mine) fold_st(static_cast<S*>(p.out) + row + i, y);
          }
        }
      }
    }
    slot = slot + 1 == kFoldWalkPairs ? 0 : slot + 1;
    buf ^= 1;
  }
  if (head) {
#pragma unroll
    for (int c = 0; c < P; ++c) {
      const int i = threadIdx.x * 4 + c * step;
      if (i < D) {
#pragma unroll
        for (int k = 0; k < LR; ++k) fold_st(win + static_cast<size_t>(k) * D + i, hist[c][k]);
      }
    }
  }
}

// LR: taps - 1 where the history fits registers (0 .. 3), -1: any number of taps, history in shared memory.
template <typename S, int LR, int V>
__global__ void __launch_bounds__(kFoldMaxWarps * 32) fold_norm_kernel(const FoldArgs p, int mode) {
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

  // every row's place in its sequence, and its statistics: inv[list index][group]
  const int list = max(p.tile_rows + L, 2 * L);
  int* place = reinterpret_cast<int*>(fold_smem);
  float* inv = fold_smem + list;
  const int groups = p.groups, gw = p.D / groups;
  float* part = inv + static_cast<size_t>(list) * groups;  // kGroupWarp: [list index][piece]; kGroupAny: [row in round][group][wpr]
  if (p.conv && L > 0 && !head)
    for (int i = threadIdx.x; i < count; i += blockDim.x) place[i] = first + i - p.cu[p.seq_of[first + i]];
  if (p.w && mode != kGroupAny) {
    // a warp takes up to 8 pieces of a row at a time, all requested together
    constexpr int B = 8;
    const int pieces = (p.D + 127) / 128, batches = (pieces + B - 1) / B;
    for (int item = warp; item < count * batches; item += n_warps) {
      const int i = item / batches, k0 = (item - i * batches) * B;
      const int row = token(i);
      Cols<V> v[B];
#pragma unroll
      for (int k = 0; k < B; ++k) {
        const int c = ((k0 + k) * 32 + lane) * 4;
        if (c < p.D) {
          v[k] = folded<S, V>(p, row, c);
        } else {
#pragma unroll
          for (int e = 0; e < V; ++e) v[k].v[e] = 0.f;
        }
      }
#pragma unroll
      for (int k = 0; k < B; ++k) {
        if (k0 + k >= pieces) break;
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < V; ++e) ss += v[k].v[e] * v[k].v[e];
        if (mode == kGroupWarp) {
          ss = warp_sum(ss);
          if (lane == 0) part[i * pieces + k0 + k] = ss;
        } else {
          ss = lanes_sum(ss, gw / 4);
          const int c = ((k0 + k) * 32 + lane) * 4;
          if (c < p.D && c % gw == 0) inv[i * groups + c / gw] = 1.f / sqrtf(ss / static_cast<float>(gw) + p.eps);
        }
      }
    }
    __syncthreads();
    if (mode == kGroupWarp) {
      const int per = gw / 128;
      for (int k = threadIdx.x; k < count * groups; k += blockDim.x) {
        const int i = k / groups, g = k - i * groups;
        float ss = 0.f;
        for (int q = 0; q < per; ++q) ss += part[i * pieces + g * per + q];
        inv[k] = 1.f / sqrtf(ss / static_cast<float>(gw) + p.eps);
      }
      __syncthreads();
    }
  } else if (p.w) {
    // group by group; several warps share a row where there are more warps than rows
    int wpr = n_warps / count;
    if (wpr < 1) wpr = 1;
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
  float* far = fold_smem + p.far_at;
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
        const int j = (head || L == 0 || !p.conv) ? 0 : place[i];
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

struct FoldLaunch {
  int n_heads, threads, mode, pieces;  // pieces > 0: the row form (walk: the walking form) with that many pieces per thread
  int walk;
  size_t smem;
};

template <typename S, int LR, int V>
int launch_fold_norm(const FoldArgs& p, const FoldLaunch& l, cudaStream_t stream) {
  auto kern = fold_norm_kernel<S, LR, V>;
  if (l.smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(l.smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  launch_pdl(kern, dim3(p.n_tiles + l.n_heads), dim3(l.threads), l.smem, stream, p, l.mode);
  return launch_status();
}

template <typename S, int LR>
int launch_fold_norm_row(const FoldArgs& p, const FoldLaunch& l, cudaStream_t stream) {
  if (l.pieces == 1) launch_pdl(fold_norm_row_kernel<S, LR, 1>, dim3(p.T), dim3(l.threads), 0, stream, p, l.mode);
  else if (l.pieces == 2) launch_pdl(fold_norm_row_kernel<S, LR, 2>, dim3(p.T), dim3(l.threads), 0, stream, p, l.mode);
  else launch_pdl(fold_norm_row_kernel<S, LR, 4>, dim3(p.T), dim3(l.threads), 0, stream, p, l.mode);
  return launch_status();
}

template <typename S, int LR, int P>
int launch_fold_norm_walk(const FoldArgs& p, const FoldLaunch& l, cudaStream_t stream) {
  auto kern = fold_norm_walk_kernel<S, LR, P>;
  const size_t smem = static_cast<size_t>(kFoldWalkPairs * 2 * P) * l.threads * (16 + 4 * sizeof(S));
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  // (no programmatic launch: a strip is a long walk, and blocks that start early pile up on few SMs)
  kern<<<dim3(p.n_tiles + l.n_heads), dim3(l.threads), smem, stream>>>(p, l.mode);
  return launch_status();
}

template <typename S, int LR>
int launch_fold_norm_walk(const FoldArgs& p, const FoldLaunch& l, cudaStream_t stream) {
  return l.pieces == 1 ? launch_fold_norm_walk<S, LR, 1>(p, l, stream) : launch_fold_norm_walk<S, LR, 2>(p, l, stream);
}

template <typename S, int V>
int dispatch_fold_norm(const FoldArgs& p, const FoldLaunch& l, cudaStream_t stream) {
  const int L = p.conv ? p.taps - 1 : 0;
  if (l.walk) {
    switch (L) {
      case 1: return launch_fold_norm_walk<S, 1>(p, l, stream);
      case 2: return launch_fold_norm_walk<S, 2>(p, l, stream);
      default: return launch_fold_norm_walk<S, 3>(p, l, stream);
    }
  }
  if (l.pieces > 0) {
    switch (L) {
      case 0: return launch_fold_norm_row<S, 0>(p, l, stream);
      case 1: return launch_fold_norm_row<S, 1>(p, l, stream);
      case 2: return launch_fold_norm_row<S, 2>(p, l, stream);
      default: return launch_fold_norm_row<S, 3>(p, l, stream);
    }
  }
  switch (L) {
    case 0: return launch_fold_norm<S, 0, V>(p, l, stream);
    case 1: return launch_fold_norm<S, 1, V>(p, l, stream);
    case 2: return launch_fold_norm<S, 2, V>(p, l, stream);
    case 3: return launch_fold_norm<S, 3, V>(p, l, stream);
    default: return launch_fold_norm<S, -1, V>(p, l, stream);
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
  const int gw = D / groups;
  const bool lanes = gw <= 64 && (gw & (gw - 1)) == 0;
  const int mode = !vec4 ? pmm::kGroupAny : gw % 128 == 0 ? pmm::kGroupWarp : lanes ? pmm::kGroupLanes : pmm::kGroupAny;
  int warps = (D / V + 31) / 32;
  if (warps > pmm::kFoldMaxWarps) warps = pmm::kFoldMaxWarps;
  const bool own_rows = L == 0 || (one_token && L <= 3);   // no block reads a row of another
  const int row_pieces = (D + 127) / 128;
  // pieces per thread of the row form: few rows spread over many threads, many rows keep their blocks small
  const int per_thread = (row_pieces + (T >= 512 ? 8 : pmm::kFoldMaxWarps) - 1) / (T >= 512 ? 8 : pmm::kFoldMaxWarps);
  pmm::FoldArgs p{h_in, h_out, a, b, sa, sb, vec, w, eps, groups, conv, taps, window, cu, slots, seq_of, rows, out, T, D,
                  0, 1, 0, 0};
  pmm::FoldLaunch l{0, 0, mode, 0, 0, 0};
  if (vec4 && own_rows && (mode != pmm::kGroupAny || !w) && per_thread <= 4) {
    l.pieces = per_thread <= 2 ? per_thread : 4;  // (a block has at most kFoldMaxWarps warps: 4 pieces are 8,192 columns)
    l.threads = (row_pieces + l.pieces - 1) / l.pieces * 32;
    PMM_DISPATCH_DTYPE(dtype, S, { return (pmm::dispatch_fold_norm<S, 4>(p, l, stream)); });
  }
  if (vec4 && L >= 1 && L <= 3 && !one_token && mode != pmm::kGroupAny && row_pieces <= pmm::FoldWalk<2>::kThreads / 32 * 2) {
    l.walk = 1;
    l.pieces = row_pieces <= pmm::FoldWalk<1>::kThreads / 32 ? 1 : 2;
    l.threads = (row_pieces + l.pieces - 1) / l.pieces * 32;
    const int blocks = 148 * (l.threads <= 384 ? 2 : 1);  // strips that are resident together
    p.tile_rows = (T + blocks - 1) / blocks;
    if (p.tile_rows < 4) p.tile_rows = 4;
    if (p.tile_rows > pmm::kFoldWalkRows - L) p.tile_rows = pmm::kFoldWalkRows - L;
    p.n_tiles = (T + p.tile_rows - 1) / p.tile_rows;
    l.n_heads = n_seq;
    PMM_DISPATCH_DTYPE(dtype, S, { return (pmm::dispatch_fold_norm<S, 4>(p, l, stream)); });
  }
  if (warps < 4) warps = 4;
  const bool heads_only = L > 0 && one_token;
  p.fold_in_heads = heads_only ? 1 : 0;
  // with a convolution a tile has as many rows (its own and the L before them) as the block has warps
  if (L > 0) p.tile_rows = warps > L + 1 ? warps - L : (L < 8 ? 8 : L);
  p.n_tiles = heads_only ? 0 : (T + p.tile_rows - 1) / p.tile_rows;
  l.n_heads = L > 0 ? n_seq : 0;
  l.threads = warps * 32;
  const int list = p.tile_rows + L > 2 * L ? p.tile_rows + L : 2 * L;
  const int parts = mode == pmm::kGroupWarp ? list * ((D + 127) / 128) : pmm::kFoldMaxWarps * groups;
  p.far_at = (list + list * groups + parts + 3) / 4 * 4;
  l.smem = (static_cast<size_t>(p.far_at) + (L > 3 ? static_cast<size_t>(L) * l.threads * V : 0)) * sizeof(float);
  if (l.smem > 200 * 1024) return PMM_ERR_BAD_ARGUMENT;
  PMM_DISPATCH_DTYPE(dtype, S, {
    if (vec4) return (pmm::dispatch_fold_norm<S, 4>(p, l, stream));
    return (pmm::dispatch_fold_norm<S, 1>(p, l, stream));
  });
  return 0;
}
