// The update rules of the matrix-state recurrences (recurrent.cu token by token, recurrent_chunked.cu in chunks) and
// what their kernels share.
#pragma once
#include "common.cuh"

namespace pmm {

// kRuleDecay:      S <- a S + k v^T;  o = S^T q,  one decay a per head, q, k, v = silu of the projections
// kRuleDelta:      S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// kRuleRetention:  kRuleDecay with q and k as projected, rotated by their positions, k times k_scale, v as projected
// kRuleWkv:        o = (S + diag(b) k v^T)^T q;  S <- diag(w) S + k v^T,  w = exp(-exp(a + a_bias)) per head, key channel
//                  and token, b (the bonus of the current token) per head and key channel
enum { kRuleDecay = 0, kRuleDelta = 1, kRuleRetention = 2, kRuleWkv = 3 };

// Rotation of q and k by position (kRuleRetention): pair f of the first rot_dims entries is (f, f + rot_dims/2) with
// `half_layout`, else (2f, 2f + 1).
struct RecRotation {
  const int* positions;
  const float* inv_freq;  // [rot_dims / 2]
  int rot_dims, half_layout;
};

// The pairs of the rows [n][stride] of q and k in shared memory turn together by the angle of their token's position
// (`q`, `k`: one row per token from token t0 on); a thread takes pairs e, e + n_threads, ...
__device__ __forceinline__ void rotate_rows(float* q, float* k, int stride, int n, int t0, const RecRotation& r, int tid,
                                            int n_threads) {
  const int half = r.rot_dims >> 1;
  for (int e = tid; e < n * half; e += n_threads) {
    const int i = e / half, f = e - i * half;
    const int a = r.half_layout ? f : 2 * f, b = r.half_layout ? f + half : 2 * f + 1;
    float s, c;
    sincosf(static_cast<float>(r.positions[t0 + i]) * r.inv_freq[f], &s, &c);
    float* qr = q + i * stride;
    float* kr = k + i * stride;
    const float qa = qr[a], qb = qr[b], ka = kr[a], kb = kr[b];
    qr[a] = qa * c - qb * s;
    qr[b] = qb * c + qa * s;
    kr[a] = ka * c - kb * s;
    kr[b] = kb * c + ka * s;
  }
}

}  // namespace pmm
