// Inputs of mixers that look one token back, and the low-rank product behind their decays.
//
// shifted_mixes: with h' the row before h of the same request (the row kept in `state` for the first token of a step,
// which is zero for a new request), n outputs  out_s = h + (h' - h) * mu_s.  Every row of h is read once per block
// that needs it (a token's block reads its own row and the one before).  What touches the state is one block's work:
// the block of a sequence's first token of the step reads it and then leaves the step's last row there.
//
// low_rank_tanh: a[t, c] = sum_r tanh(z[t, r]) w[c, r] in float, for steps of few tokens and for float operands.
#include "common.cuh"

namespace pmm {

constexpr int kMixThreads = 256;
constexpr int kMixMax = 8;

template <typename S, int VEC>
struct RowPiece;
template <typename S>
struct RowPiece<S, 1> {
  static __device__ __forceinline__ void load(const S* p, float (&v)[1]) { v[0] = ldf(p); }
  static __device__ __forceinline__ void store(S* p, const float (&v)[1]) { stf(p, v[0]); }
};
template <typename S>
struct RowPiece<S, 4> {
  static __device__ __forceinline__ void load(const S* p, float (&v)[4]) {
    const float4 x = ldf4(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
  }
  static __device__ __forceinline__ void store(S* p, const float (&v)[4]) { stf4(p, make_float4(v[0], v[1], v[2], v[3])); }
};

// A block takes the columns blockIdx.y * kMixThreads * VEC .. of `tokens` consecutive rows from blockIdx.x * tokens on.
template <typename S, int VEC>
__global__ void __launch_bounds__(kMixThreads)
    shifted_mixes_kernel(const S* __restrict__ x, long long ld_x, const float* __restrict__ mu, int n_mixes,
                         float* __restrict__ state, const int* __restrict__ cu, const int* __restrict__ slots,
                         const int* __restrict__ seq_of, S* __restrict__ out, long long mix_stride, int T, int D, int tokens) {
  using P = RowPiece<S, VEC>;
  using PF = RowPiece<float, VEC>;
  const int c = (blockIdx.y * kMixThreads + threadIdx.x) * VEC;
  float m[kMixMax][VEC];
  pdl_launch_dependents();
#pragma unroll
  for (int s = 0; s < kMixMax; ++s)  // (the mixes' weights are constants: read before the wait)
    if (s < n_mixes && c < D) PF::load(mu + static_cast<size_t>(s) * D + c, m[s]);
  pdl_wait();
  if (c >= D) return;
  const int t_begin = blockIdx.x * tokens, t_end = min(T, t_begin + tokens);
  float before[VEC];
  bool have = false;  // `before` holds row t - 1
  for (int t = t_begin; t < t_end; ++t) {
    const int seq = seq_of[t], first = cu[seq];
    float h[VEC];
    P::load(x + static_cast<long long>(t) * ld_x + c, h);
    if (t == first) {
      float* st = state + static_cast<size_t>(slots[seq]) * D + c;
      PF::load(st, before);
      const int last = cu[seq + 1] - 1;
      float hl[VEC];
      P::load(x + static_cast<long long>(last) * ld_x + c, hl);
      PF::store(st, hl);
    } else if (!have) {
      P::load(x + static_cast<long long>(t - 1) * ld_x + c, before);
    }
#pragma unroll
    for (int s = 0; s < kMixMax; ++s) {
      if (s < n_mixes) {
        float y[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = h[e] + (before[e] - h[e]) * m[s][e];
        P::store(out + s * mix_stride + static_cast<long long>(t) * D + c, y);
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) before[e] = h[e];
    have = true;
  }
}

// ---- a = tanh(z) w^T: a block takes 32 channels and up to 16 tokens, 8 at a time; z [T, R], w [C, R]
constexpr int kLrThreads = 256;
constexpr int kLrChannels = 32;  // channels per block, 8 lanes each

template <typename S>
__global__ void __launch_bounds__(kLrThreads)
    low_rank_tanh_kernel(const S* __restrict__ z, long long ld_z, const S* __restrict__ w, float* __restrict__ a, int T, int C,
                         int R, int tokens) {
  extern __shared__ float sm[];  // [tokens][R] tanh(z)
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.y * tokens, n = min(tokens, T - t0);
  for (int e = threadIdx.x; e < n * R; e += kLrThreads) {
    const int t = e / R, r = e - t * R;
    sm[e] = tanhf(ldf(z + static_cast<long long>(t0 + t) * ld_z + r));
  }
  __syncthreads();
  const int lane8 = threadIdx.x & 7;
  const int c = blockIdx.x * kLrChannels + (threadIdx.x >> 3);
  const S* row = w + static_cast<size_t>(c < C ? c : 0) * R;
  for (int tb = 0; tb < n; tb += 8) {
    float acc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = 0.f;
    for (int r = lane8; r < R; r += 8) {
      const float wv = ldf(row + r);
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (tb + j < n) acc[j] += sm[(tb + j) * R + r] * wv;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], 1);
      acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], 2);
      acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], 4);
      if (lane8 == j && tb + j < n && c < C) a[static_cast<size_t>(t0 + tb + j) * C + c] = acc[j];
    }
  }
}

}  // namespace pmm

// x [T, D] rows of stride ld_x; mu [n_mixes, D] floats; state [slots, D] floats; out: mix s at out + s * mix_stride,
// rows of D.  At most 8 mixes.
PMM_EXPORT int pmm_shifted_mixes(const void* x, long long ld_x, const float* mu, int n_mixes, float* state, const int* cu,
                                 const int* slots, const int* seq_of, void* out, long long mix_stride, int T, int D, int dtype,
                                 cudaStream_t stream) {
  if (T <= 0) return 0;
  if (D <= 0 || n_mixes < 1 || n_mixes > pmm::kMixMax || !state) return PMM_ERR_BAD_ARGUMENT;
  auto aligned = [](const void* p, size_t n) { return reinterpret_cast<uintptr_t>(p) % n == 0; };
  const bool vec = D % 4 == 0 && ld_x % 4 == 0 && mix_stride % 4 == 0 && aligned(x, 16) && aligned(mu, 16) && aligned(state, 16) &&
                   aligned(out, 16);
  const int cols = pmm::kMixThreads * (vec ? 4 : 1);
  const int gy = (D + cols - 1) / cols;
  // rows per block: two in steps of many tokens, so that half of the rows before come from registers
  const int tokens = static_cast<long long>(T) * gy >= 4 * 148 * 8 ? 4 : (static_cast<long long>(T) * gy >= 2 * 148 * 4 ? 2 : 1);
  const dim3 grid((T + tokens - 1) / tokens, gy);
  PMM_DISPATCH_DTYPE(dtype, S, {
    auto kern = vec ? pmm::shifted_mixes_kernel<S, 4> : pmm::shifted_mixes_kernel<S, 1>;
    pmm::launch_pdl(kern, grid, dim3(pmm::kMixThreads), 0, stream, static_cast<const S*>(x), ld_x, mu, n_mixes, state, cu, slots,
                    seq_of, static_cast<S*>(out), mix_stride, T, D, tokens);
  });
  return pmm::launch_status();
}

// z [T, R] rows of stride ld_z, w [C, R] of one storage type; a [T, C] floats.
PMM_EXPORT int pmm_low_rank_tanh(const void* z, long long ld_z, const void* w, float* a, int T, int C, int R, int dtype,
                                 cudaStream_t stream) {
  if (T <= 0) return 0;
  if (C <= 0 || R <= 0 || R > 2048) return PMM_ERR_BAD_ARGUMENT;
  int tokens = 16;  // (more of them a block: less of w read twice, but fewer blocks)
  while (tokens > 8 && sizeof(float) * static_cast<size_t>(tokens) * R > 40 * 1024) tokens /= 2;
  const size_t smem = sizeof(float) * static_cast<size_t>(tokens) * R;
  const dim3 grid((C + pmm::kLrChannels - 1) / pmm::kLrChannels, (T + tokens - 1) / tokens);
  if (grid.y > 65535) return PMM_ERR_BAD_ARGUMENT;
  PMM_DISPATCH_DTYPE(dtype, S, {
    auto kern = pmm::low_rank_tanh_kernel<S>;
    if (smem > 48 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
      if (e != cudaSuccess) return static_cast<int>(e);
    }
    pmm::launch_pdl(kern, grid, dim3(pmm::kLrThreads), smem, stream, static_cast<const S*>(z), ld_z, static_cast<const S*>(w), a,
                    T, C, R, tokens);
  });
  return pmm::launch_status();
}
