// Rotation on part of every head, and the write into the cache pages, for heads whose key size d and
// value size dv differ.
//
// The first rot_dims entries of every query and key head are rotated in pairs (x, y): at position p they
// become (x cos a - y sin a, y cos a + x sin a) with a = p * inv_freq[i].  Pair i is entries (2i, 2i+1)
// (neighbouring pairs) or entries (i, i + rot_dims/2) (half layout: the first half of the rotated
// part against its second half); entries from rot_dims on pass unchanged; values are not rotated.
// A bias per channel (float, optional) is added to q, k and v as they are read.  Positions, angles, sines and cosines are
// float.  Queries go to q_out [T, H*Dp], keys and values into their page
// [page, plane, page_size, G*Dp]: all heads are laid out Dp = max(d, dv) rounded up wide, padded
// with zeros, so that one attention kernel of head size Dp serves both sizes (zeros add nothing to
// a score, and the padded value columns come out zero and are dropped by the output projection's
// operand view).  v_norm_eps >= 0: every value head is divided by its own root mean square
// (v / sqrt(mean(v^2) + eps) over its dv entries, no weight, float) before it is written.
#include "common.cuh"

namespace pmm {

constexpr int kRopeMaxPairs = 128;  // rot_dims <= 256
constexpr int kRopeMaxGroups = 256;  // key/value heads whose values are normed

// `sn`, `cs`: the token's sines and cosines per rotated pair (shared memory, made once a token).
template <typename S>
__device__ __forceinline__ float rotated(const S* __restrict__ head, const float* __restrict__ bias, int i, int rot_dims,
                                         const float* __restrict__ sn_t, const float* __restrict__ cs_t, int half_layout,
                                         const float* __restrict__ norm_w = nullptr, float inv = 1.f) {
  const float x = (ldf(head + i) + (bias ? bias[i] : 0.f)) * (norm_w ? inv * norm_w[i] : 1.f);
  if (i >= rot_dims) return x;
  const int half = rot_dims >> 1;
  const bool second = half_layout ? i >= half : (i & 1);
  const int j = half_layout ? (second ? i - half : i + half) : (i ^ 1);
  const int f = half_layout ? (second ? i - half : i) : (i >> 1);
  const float other = (ldf(head + j) + (bias ? bias[j] : 0.f)) * (norm_w ? inv * norm_w[j] : 1.f);
  const float sn = sn_t[f], cs = cs_t[f];
  return second ? x * cs + other * sn : x * cs - other * sn;
}

template <typename S>
__global__ void __launch_bounds__(256)
    rope_pairs_store_kernel(const S* __restrict__ q, long long ld_q, const S* __restrict__ k, long long ld_k,
                            const S* __restrict__ v, long long ld_v, const float* __restrict__ inv_freq,
                            const int* __restrict__ positions, const int* __restrict__ seq_of,
                            const int* __restrict__ block_table, int max_blocks, S* __restrict__ pool,
                            int page_size, S* __restrict__ q_out, int H, int G, int d, int dv, int Dp,
                            int rot_dims, int half_layout, const float* __restrict__ q_bias,
                            const float* __restrict__ k_bias, const float* __restrict__ v_bias,
                            const float* __restrict__ q_norm_w, const float* __restrict__ k_norm_w, float norm_eps,
                            float v_norm_eps) {
  __shared__ float sn_t[kRopeMaxPairs], cs_t[kRopeMaxPairs];
  __shared__ float inv_v[kRopeMaxGroups];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int pos = positions[t];
  const float fpos = static_cast<float>(pos);
  for (int f = threadIdx.x; f < rot_dims / 2; f += blockDim.x) sincosf(fpos * inv_freq[f], &sn_t[f], &cs_t[f]);
  // q_norm_w / k_norm_w: all query rows of the token, and all its key rows, are divided by their root mean
  // square (over the whole projection, before it is cut into heads) and multiplied by the weight, before rotation
  float inv_q = 1.f, inv_k = 1.f;
  if (q_norm_w) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < H * d; i += blockDim.x) {
      const float x = ldf(q + static_cast<long long>(t) * ld_q + i) + (q_bias ? q_bias[i] : 0.f);
      ss += x * x;
    }
    inv_q = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(H * d) + norm_eps);
  }
  if (k_norm_w) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < G * d; i += blockDim.x) {
      const float x = ldf(k + static_cast<long long>(t) * ld_k + i) + (k_bias ? k_bias[i] : 0.f);
      ss += x * x;
    }
    inv_k = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(G * d) + norm_eps);
  }
  if (v_norm_eps >= 0.f) {
    const int lane = threadIdx.x & 31;
    for (int g = threadIdx.x >> 5; g < G; g += blockDim.x >> 5) {  // a warp per value head
      float ss = 0.f;
      for (int i = lane; i < dv; i += 32) {
        const float x = ldf(v + static_cast<long long>(t) * ld_v + g * dv + i) + (v_bias ? v_bias[g * dv + i] : 0.f);
        ss += x * x;
      }
      ss = warp_sum(ss);
      if (lane == 0) inv_v[g] = 1.f / sqrtf(ss / static_cast<float>(dv) + v_norm_eps);
    }
  }
  __syncthreads();
  const int n_q = H * Dp, n_kv = G * Dp;
  const int page = block_table[static_cast<size_t>(seq_of[t]) * max_blocks + pos / page_size];
  S* k_row = pool + (static_cast<size_t>(page) * 2 * page_size + pos % page_size) * n_kv;
  S* v_row = k_row + static_cast<size_t>(page_size) * n_kv;
  for (int e = threadIdx.x; e < n_q + 2 * n_kv; e += blockDim.x) {
    if (e < n_q) {
      const int h = e / Dp, i = e - h * Dp;
      const float val = i < d ? rotated(q + static_cast<long long>(t) * ld_q + h * d, q_bias ? q_bias + h * d : nullptr, i, rot_dims,
                                        sn_t, cs_t, half_layout, q_norm_w ? q_norm_w + h * d : nullptr, inv_q) : 0.f;
      stf(q_out + static_cast<size_t>(t) * n_q + e, val);
    } else if (e < n_q + n_kv) {
      const int c = e - n_q, g = c / Dp, i = c - g * Dp;
      const float val = i < d ? rotated(k + static_cast<long long>(t) * ld_k + g * d, k_bias ? k_bias + g * d : nullptr, i, rot_dims,
                                        sn_t, cs_t, half_layout, k_norm_w ? k_norm_w + g * d : nullptr, inv_k) : 0.f;
      stf(k_row + c, val);
    } else {
      const int c = e - n_q - n_kv, g = c / Dp, i = c - g * Dp;
      float val = i < dv ? ldf(v + static_cast<long long>(t) * ld_v + g * dv + i) + (v_bias ? v_bias[g * dv + i] : 0.f) : 0.f;
      if (v_norm_eps >= 0.f) val *= inv_v[g];
      stf(v_row + c, val);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------
// The same preparation with a norm per head: bias, the head's RMS norm (with a weight that all heads share, without
// one, or none), rotation with sines and cosines times an amplitude, and values that are mixed with the values an
// earlier layer left for the same tokens,  v <- (1 - l) v + l v0.  A warp takes one head row (a query, key or value
// head of a token): it keeps the row in registers for the norm, in its own piece of shared memory for the rotation's
// partner entries, and writes the padded row.  Blocks of 8 warps; the rows of a token are spread over gridDim.y.
constexpr int kHeadRopeWarps = 8;
constexpr int kHeadRopeMaxDim = 256;
constexpr int kHeadRopePer = kHeadRopeMaxDim / 32;

struct HeadRopeArgs {
  const void *q, *k, *v;
  long long ld_q, ld_k, ld_v;
  const float* inv_freq;
  const int *positions, *seq_of, *block_table;
  int max_blocks, page_size;
  void *pool, *q_out;
  int H, G, d, dv, Dp, rot_dims, half_layout;
  float amplitude;
  const float *q_bias, *k_bias, *v_bias;
  float norm_eps;                  // below zero: no norm
  const float *q_w, *k_w;          // [d] or nullptr
  void* values;                    // [T, G*dv] or nullptr: the earlier layer's values (mix given) or where to leave these
  const float* mix;                // one value, or nullptr
};

template <typename S>
__global__ void __launch_bounds__(kHeadRopeWarps * 32)
    head_norm_rope_store_kernel(const HeadRopeArgs p) {
  __shared__ float sn_t[kRopeMaxPairs], cs_t[kRopeMaxPairs];
  __shared__ float rows[kHeadRopeWarps][kHeadRopeMaxDim];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.positions[t];
  const float fpos = static_cast<float>(pos);
  const int half = p.rot_dims >> 1;
  const int n_rows = p.H + 2 * p.G;
  // (a block of value rows alone turns nothing)
  if (static_cast<int>(blockIdx.y) * kHeadRopeWarps < p.H + p.G)
    for (int f = threadIdx.x; f < half; f += blockDim.x) {
      float s, c;
      sincosf(fpos * p.inv_freq[f], &s, &c);
      sn_t[f] = s * p.amplitude;
      cs_t[f] = c * p.amplitude;
    }
  __syncthreads();
  const int row = blockIdx.y * kHeadRopeWarps + warp;
  if (row >= n_rows) return;
  S* page_row = nullptr;
  if (row >= p.H) {
    const int page = p.block_table[static_cast<size_t>(p.seq_of[t]) * p.max_blocks + pos / p.page_size];
    page_row = static_cast<S*>(p.pool) + (static_cast<size_t>(page) * 2 * p.page_size + pos % p.page_size) * (p.G * p.Dp);
  }
  if (row >= p.H + p.G) {  // ---- a value head
    const int g = row - p.H - p.G;
    const S* src = static_cast<const S*>(p.v) + static_cast<long long>(t) * p.ld_v + g * p.dv;
    S* vals = p.values ? static_cast<S*>(p.values) + (static_cast<size_t>(t) * p.G + g) * p.dv : nullptr;
    S* dst = page_row + static_cast<size_t>(p.page_size) * (p.G * p.Dp) + g * p.Dp;
    const float l = p.mix ? *p.mix : 0.f;
    for (int i = lane; i < p.Dp; i += 32) {
      float x = 0.f;
      if (i < p.dv) {
        x = ldf(src + i) + (p.v_bias ? p.v_bias[g * p.dv + i] : 0.f);
        if (p.mix) x = (1.f - l) * x + l * ldf(vals + i);
        else if (vals) stf(vals + i, x);
      }
      stf(dst + i, x);
    }
    return;
  }
  const bool is_q = row < p.H;
  const int h = is_q ? row : row - p.H;
  const S* src = is_q ? static_cast<const S*>(p.q) + static_cast<long long>(t) * p.ld_q + h * p.d
                      : static_cast<const S*>(p.k) + static_cast<long long>(t) * p.ld_k + h * p.d;
  const float* bias = is_q ? p.q_bias : p.k_bias;
  const float* w = is_q ? p.q_w : p.k_w;
  float x[kHeadRopePer];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < kHeadRopePer; ++j) {
    const int i = lane + 32 * j;
    x[j] = 0.f;
    if (i < p.d) x[j] = ldf(src + i) + (bias ? bias[h * p.d + i] : 0.f);
    ss += x[j] * x[j];
  }
  if (p.norm_eps >= 0.f) {
    const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(p.d) + p.norm_eps);
#pragma unroll
    for (int j = 0; j < kHeadRopePer; ++j) {
      const int i = lane + 32 * j;
      if (i < p.d) x[j] *= w ? inv * w[i] : inv;
    }
  }
  if (half > 0) {
#pragma unroll
    for (int j = 0; j < kHeadRopePer; ++j) {
      const int i = lane + 32 * j;
      if (i < p.rot_dims) rows[warp][i] = x[j];
    }
    __syncwarp();
#pragma unroll
    for (int j = 0; j < kHeadRopePer; ++j) {
      const int i = lane + 32 * j;
      if (i < p.rot_dims) {
        const bool second = p.half_layout ? i >= half : (i & 1);
        const int other = p.half_layout ? (second ? i - half : i + half) : (i ^ 1);
        const int f = p.half_layout ? (second ? i - half : i) : (i >> 1);
        const float y = rows[warp][other];
        x[j] = second ? x[j] * cs_t[f] + y * sn_t[f] : x[j] * cs_t[f] - y * sn_t[f];
      }
    }
  }
  S* dst = is_q ? static_cast<S*>(p.q_out) + (static_cast<size_t>(t) * p.H + h) * p.Dp : page_row + h * p.Dp;
#pragma unroll
  for (int j = 0; j < kHeadRopePer; ++j) {
    const int i = lane + 32 * j;
    if (i < p.Dp) stf(dst + i, x[j]);  // (entries from d on are zero)
  }
}

// The same for heads of an even size whose turning pairs are neighbours (or that do not turn): a lane holds the pairs
// lane, lane + 32, ... of a head, so the partner is its own and the sines and cosines, made once, serve every row of the
// token that the warp takes (rows warp, warp + WARPS, ..., all of them loaded before the first is used).
template <typename S, int NP, int ROWS>  // NP pairs per lane: heads of up to 64 NP entries
__global__ void __launch_bounds__(kHeadRopeWarps * 32)
    head_norm_rope_pairs_kernel(const HeadRopeArgs p) {
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_rows = p.H + 2 * p.G, half = p.rot_dims >> 1;
  const int first = (blockIdx.y * kHeadRopeWarps + warp) * ROWS;
  pdl_wait();
  if (first >= n_rows) return;
  const int pos = p.positions[t];
  float2 x[ROWS][NP];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int row = first + r;
    const bool is_q = row < p.H, is_v = row >= p.H + p.G;
    const int h = is_q ? row : is_v ? row - p.H - p.G : row - p.H;
    const int width = is_v ? p.dv : p.d;
    const S* src = (is_q ? static_cast<const S*>(p.q) + static_cast<long long>(t) * p.ld_q
                         : is_v ? static_cast<const S*>(p.v) + static_cast<long long>(t) * p.ld_v
                                : static_cast<const S*>(p.k) + static_cast<long long>(t) * p.ld_k) + h * width;
    const float* bias = is_q ? p.q_bias : is_v ? p.v_bias : p.k_bias;
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int i = 2 * (lane + 32 * j);
      x[r][j] = make_float2(0.f, 0.f);
      if (row < n_rows && i < width) {
        x[r][j] = ldf2(src + i);
        if (bias) {
          const float2 b = ldf2(bias + h * width + i);
          x[r][j].x += b.x;
          x[r][j].y += b.y;
        }
      }
    }
  }
  float2 turn[NP];  // cosine, sine
  if (first < p.H + p.G) {
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int f = lane + 32 * j;
      turn[j] = make_float2(1.f, 0.f);
      if (f < half) {
        float s, c;
        sincosf(static_cast<float>(pos) * p.inv_freq[f], &s, &c);
        turn[j] = make_float2(c * p.amplitude, s * p.amplitude);
      }
    }
  }
  S* page_row = nullptr;
  if (first + ROWS > p.H) {
    const int page = p.block_table[static_cast<size_t>(p.seq_of[t]) * p.max_blocks + pos / p.page_size];
    page_row = static_cast<S*>(p.pool) + (static_cast<size_t>(page) * 2 * p.page_size + pos % p.page_size) * (p.G * p.Dp);
  }
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int row = first + r;
    if (row >= n_rows) return;
    if (row >= p.H + p.G) {
      const int g = row - p.H - p.G;
      S* vals = p.values ? static_cast<S*>(p.values) + (static_cast<size_t>(t) * p.G + g) * p.dv : nullptr;
      S* dst = page_row + static_cast<size_t>(p.page_size) * (p.G * p.Dp) + g * p.Dp;
      const float l = p.mix ? *p.mix : 0.f;
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        const int i = 2 * (lane + 32 * j);
        if (i < p.dv) {
          if (p.mix) {
            const float2 y = ldf2(vals + i);
            x[r][j] = make_float2((1.f - l) * x[r][j].x + l * y.x, (1.f - l) * x[r][j].y + l * y.y);
          } else if (vals) {
            stf2(vals + i, x[r][j]);
          }
        }
        if (i < p.Dp) stf2(dst + i, x[r][j]);
      }
      continue;
    }
    const bool is_q = row < p.H;
    const int h = is_q ? row : row - p.H;
    if (p.norm_eps >= 0.f) {
      const float* w = is_q ? p.q_w : p.k_w;
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < NP; ++j) ss += x[r][j].x * x[r][j].x + x[r][j].y * x[r][j].y;
      const float inv = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(p.d) + p.norm_eps);
#pragma unroll
      for (int j = 0; j < NP; ++j) {
        const int i = 2 * (lane + 32 * j);
        float2 g = make_float2(1.f, 1.f);
        if (w && i < p.d) g = ldf2(w + i);
        x[r][j] = make_float2(x[r][j].x * inv * g.x, x[r][j].y * inv * g.y);
      }
    }
    S* dst = is_q ? static_cast<S*>(p.q_out) + (static_cast<size_t>(t) * p.H + h) * p.Dp : page_row + h * p.Dp;
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int i = 2 * (lane + 32 * j);
      const float2 y = make_float2(x[r][j].x * turn[j].x - x[r][j].y * turn[j].y, x[r][j].y * turn[j].x + x[r][j].x * turn[j].y);
      if (i < p.Dp) stf2(dst + i, y);  // (entries from d on are zero; what does not turn has cosine one, sine zero)
    }
  }
}

template <typename S, int NP>
void launch_head_rope_pairs(const HeadRopeArgs& a, int T, cudaStream_t stream) {
  const int n_rows = a.H + 2 * a.G;
  const int warps1 = n_rows, warps2 = (n_rows + 1) / 2;
  if (T >= 128)  // enough tokens to fill the GPU: two rows a warp
    launch_pdl(head_norm_rope_pairs_kernel<S, NP, 2>, dim3(T, (warps2 + kHeadRopeWarps - 1) / kHeadRopeWarps),
               dim3(kHeadRopeWarps * 32), 0, stream, a);
  else
    launch_pdl(head_norm_rope_pairs_kernel<S, NP, 1>, dim3(T, (warps1 + kHeadRopeWarps - 1) / kHeadRopeWarps),
               dim3(kHeadRopeWarps * 32), 0, stream, a);
}

}  // namespace pmm

// q [T, H*d], k [T, G*d], v [T, G*dv] rows of stride ld; inv_freq [rot_dims/2] floats (may be nullptr when
// rot_dims is 0); pool [pages, 2, page_size, G*Dp]; q_out [T, H*Dp]; q_bias [H*d], k_bias [G*d], v_bias [G*dv]
// floats or nullptr; q_norm_w [H*d], k_norm_w [G*d] floats or nullptr: an RMS norm over the token's whole query
// (key) projection before rotation, eps inside the root; v_norm_eps >= 0: every value head over its own root mean
// square (at most kRopeMaxGroups heads).
PMM_EXPORT int pmm_rope_pairs_store(const void* q, long long ld_q, const void* k, long long ld_k, const void* v,
                                    long long ld_v, const float* inv_freq, const int* positions, const int* seq_of,
                                    const int* block_table, int max_blocks, void* pool, int page_size, void* q_out,
                                    int T, int H, int G, int d, int dv, int Dp, int rot_dims, int half_layout,
                                    const float* q_bias, const float* k_bias, const float* v_bias,
                                    const float* q_norm_w, const float* k_norm_w, float norm_eps, float v_norm_eps,
                                    int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || d <= 0 || dv <= 0 || Dp < d || Dp < dv || rot_dims < 0 || rot_dims > d || rot_dims % 2 ||
      (v_norm_eps >= 0.f && G > pmm::kRopeMaxGroups) || rot_dims > 2 * pmm::kRopeMaxPairs || (rot_dims > 0 && !inv_freq) || page_size <= 0)
    return PMM_ERR_BAD_ARGUMENT;
  PMM_DISPATCH_DTYPE(dtype, S, pmm::launch_pdl(pmm::rope_pairs_store_kernel<S>, dim3(T), dim3(256), 0, stream,
                                               static_cast<const S*>(q), ld_q, static_cast<const S*>(k), ld_k,
                                               static_cast<const S*>(v), ld_v, inv_freq, positions, seq_of,
                                               block_table, max_blocks, static_cast<S*>(pool), page_size,
                                               static_cast<S*>(q_out), H, G, d, dv, Dp, rot_dims, half_layout, q_bias,
                                               k_bias, v_bias, q_norm_w, k_norm_w, norm_eps, v_norm_eps));
  return pmm::launch_status();
}

// q [T, H*d], k [T, G*d], v [T, G*dv] rows of stride ld; pool [pages, 2, page_size, G*Dp]; q_out [T, H*Dp]; biases,
// norm weights [d] floats or nullptr; norm_eps below zero: no norm; values [T, G*dv] or nullptr, mix one float or
// nullptr (values are read where mix is given and written where it is not).  Dp up to 256.
PMM_EXPORT int pmm_head_norm_rope_store(const void* q, long long ld_q, const void* k, long long ld_k, const void* v,
                                        long long ld_v, const float* inv_freq, const int* positions, const int* seq_of,
                                        const int* block_table, int max_blocks, void* pool, int page_size, void* q_out,
                                        int T, int H, int G, int d, int dv, int Dp, int rot_dims, int half_layout,
                                        float amplitude, const float* q_bias, const float* k_bias, const float* v_bias,
                                        float norm_eps, const float* q_w, const float* k_w, void* values, const float* mix,
                                        int dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || d <= 0 || dv <= 0 || Dp < d || Dp < dv || Dp > pmm::kHeadRopeMaxDim || rot_dims < 0 || rot_dims > d ||
      rot_dims % 2 || (rot_dims > 0 && !inv_freq) || page_size <= 0 || (mix && !values))
    return PMM_ERR_BAD_ARGUMENT;
  const pmm::HeadRopeArgs a{q, k, v, ld_q, ld_k, ld_v, inv_freq, positions, seq_of, block_table, max_blocks, page_size,
                            pool, q_out, H, G, d, dv, Dp, rot_dims, half_layout, amplitude, q_bias, k_bias, v_bias,
                            norm_eps, q_w, k_w, values, mix};
  const size_t unit = dtype == PMM_DTYPE_BF16 ? 4 : 8;
  auto even = [](const void* ptr, size_t bytes) { return reinterpret_cast<uintptr_t>(ptr) % bytes == 0; };
  if ((rot_dims == 0 || !half_layout) && d % 2 == 0 && dv % 2 == 0 && Dp % 2 == 0 && ld_q % 2 == 0 && ld_k % 2 == 0 && ld_v % 2 == 0 &&
      even(q, unit) && even(k, unit) && even(v, unit) && even(pool, unit) && even(q_out, unit) && even(values, unit) &&
      even(q_bias, 8) && even(k_bias, 8) && even(v_bias, 8) && even(q_w, 8) && even(k_w, 8)) {
    PMM_DISPATCH_DTYPE(dtype, S, {
      if (Dp <= 64) pmm::launch_head_rope_pairs<S, 1>(a, T, stream);
      else if (Dp <= 128) pmm::launch_head_rope_pairs<S, 2>(a, T, stream);
      else pmm::launch_head_rope_pairs<S, 4>(a, T, stream);
    });
    return pmm::launch_status();
  }
  const dim3 grid(T, (H + 2 * G + pmm::kHeadRopeWarps - 1) / pmm::kHeadRopeWarps);
  PMM_DISPATCH_DTYPE(dtype, S, pmm::launch_pdl(pmm::head_norm_rope_store_kernel<S>, grid, dim3(pmm::kHeadRopeWarps * 32), 0, stream, a));
  return pmm::launch_status();
}
