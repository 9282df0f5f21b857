// What the recurrences with a decay per head share (ssd.cu, ssd_tc.cu): sizes, and the pass that turns the ends of a
// sequence's segments into the states they start from.
#pragma once
#include "common.cuh"

namespace dlgo {

// where a sequence's inputs of earlier steps lie: entry j of taps - 1, oldest first
struct SsdShape {
  int H, G, N, P, taps;
  __host__ __device__ int inner() const { return H * P; }
  __host__ __device__ int channels() const { return H * P + 2 * G * N; }
  __host__ __device__ long long conv_off() const { return (long long)H * N * P; }
};

// seg[j] <- the state segment j starts from.  A block row per first segment of a sequence, a thread per W neighbouring
// elements of the state; the ends of up to eight segments are fetched together.
template <int W>
__global__ void __launch_bounds__(256)
ssd_carry_kernel(const int* __restrict__ tiles, int n_tiles, const int* __restrict__ seq_slot, const float* state,
                 long long state_ld, float* seg, const float* seg_decay, SsdShape s) {
  pdl_launch_dependents();
  const int j0 = blockIdx.y;
  const int seq = tiles[j0 * 3];
  if (j0 > 0 && tiles[(j0 - 1) * 3] == seq) return;
  const long long per_head = (long long)s.N * s.P, total = per_head * s.H;
  const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * W;
  if (i >= total) return;
  const int h = (int)(i / per_head);                               // (W = 4 only where a head's numbers are a multiple of 4)
  pdl_wait();
  float S[W];
  const float* st = state + (size_t)seq_slot[seq] * state_ld + i;
#pragma unroll
  for (int k = 0; k < W; ++k) S[k] = st[k];
  for (int jb = j0; jb < n_tiles && tiles[jb * 3] == seq; jb += 8) {
    float L[8][W], F[8];
    int n = 0;
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      const int j = jb + u;
      const bool in = j < n_tiles && tiles[j * 3] == seq;
      n += in;
      const bool more = in && j + 1 < n_tiles && tiles[(j + 1) * 3] == seq;   // (a sequence's last segment left no end)
      F[u] = more ? seg_decay[(size_t)j * s.H + h] : 0.f;
      if (W == 4) {
        const float4 v = more ? *reinterpret_cast<const float4*>(seg + (size_t)j * total + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        L[u][0] = v.x; L[u][1 % W] = v.y; L[u][2 % W] = v.z; L[u][3 % W] = v.w;
      } else {
        L[u][0] = more ? seg[(size_t)j * total + i] : 0.f;
      }
    }
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      if (u < n) {
        float* dst = seg + (size_t)(jb + u) * total + i;
        if (W == 4) *reinterpret_cast<float4*>(dst) = make_float4(S[0], S[1 % W], S[2 % W], S[3 % W]);
        else dst[0] = S[0];
#pragma unroll
        for (int k = 0; k < W; ++k) S[k] = fmaf(F[u], S[k], L[u][k]);
      }
    }
  }
}

// the carry over `n_tiles` segments whose ends (a head's [N, P] numbers each) lie in seg, their decays in seg_decay
inline int launch_ssd_carry(const int* tiles, int n_tiles, const int* seq_slot, const float* state, long long state_ld,
                            float* seg, const float* seg_decay, SsdShape s, cudaStream_t stream) {
  const long long total = (long long)s.H * s.N * s.P;
  const bool four = ((long long)s.N * s.P) % 4 == 0 && (state_ld & 3) == 0 && ((uintptr_t)state & 15) == 0 &&
                    ((uintptr_t)seg & 15) == 0;
  const long long items = four ? total / 4 : total;
  const dim3 grid((unsigned)((items + 255) / 256), n_tiles);
  if (four) launch_kernel(ssd_carry_kernel<4>, grid, dim3(256), 0, stream, tiles, n_tiles, seq_slot, state, state_ld, seg, seg_decay, s);
  else launch_kernel(ssd_carry_kernel<1>, grid, dim3(256), 0, stream, tiles, n_tiles, seq_slot, state, state_ld, seg, seg_decay, s);
  return launch_status();
}

}  // namespace dlgo
