// Combining the per-slice partial results of split-KV attention (shared by the attention kernels).
#pragma once
#include <math.h>

#include "common.cuh"

namespace dlgo {

// A sink is a number per head whose exponential joins the softmax's denominator once; it has no key and no value.
// (a, l): a weighted sum and its denominator, both relative to the maximum m; afterwards relative to the larger of
// m and the sink, with the sink in l.  `sink` null: no sink.
__device__ __forceinline__ void join_sink(float& a, float& l, float m, const float* __restrict__ sink, int head) {
  if (sink == nullptr) return;
  const float s = sink[head], top = fmaxf(m, s), c = expf(m - top);
  a *= c;
  l = fmaf(l, c, expf(s - top));
}

// out[token, head, :] = sum_s w_s acc_s / (sum_s w_s l_s + the sink's share) with w_s = exp(m_s - max m)
template <typename T>
__global__ void attention_combine_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml,
                                         T* __restrict__ out, int ldo, int Hq, int hd, int n_splits,
                                         const float* __restrict__ sink) {
  pdl_launch_dependents();
  pdl_wait();
  const int token = blockIdx.x, head = blockIdx.y;
  const size_t o = ((size_t)token * Hq + head) * n_splits;
  float m = -INFINITY;
  for (int s = 0; s < n_splits; ++s) m = fmaxf(m, part_ml[(o + s) * 2]);
  float denom = 0.f;
  for (int s = 0; s < n_splits; ++s) {
    const float ms = part_ml[(o + s) * 2];
    if (ms != -INFINITY) denom += expf(ms - m) * part_ml[(o + s) * 2 + 1];
  }
  for (int d = threadIdx.x; d < hd; d += blockDim.x) {
    float a = 0.f;
    for (int s = 0; s < n_splits; ++s) {
      const float ms = part_ml[(o + s) * 2];
      if (ms != -INFINITY) a = fmaf(expf(ms - m), part_acc[(o + s) * hd + d], a);
    }
    float l = denom;
    join_sink(a, l, m, sink, head);
    out[(size_t)token * ldo + (size_t)head * hd + d] = from_float<T>(a / l);
  }
}

}  // namespace dlgo
