// A head's state [N, P] in the registers of a block, shared by the kernels that walk a recurrence S <- f S + d B x^T token
// by token: a thread holds 16 rows x 4 columns.  RS neighbouring lanes share four columns; lane r of them holds rows
// 4 (i RS + r) .. + 3 for i = 0 .. 3, and their parts of S^T C meet by shuffles.  N up to 512; rows beyond N and columns
// beyond P are computed on zeros and not stored.
#pragma once
#include "common.cuh"

namespace dlgo {

// y[k] of the RS lanes that share four columns brought together: afterwards lane r < min(RS, 4) holds the sum of
// columns (4 / min(RS, 4)) * r .. in y[0 ..].
template <int RS>
__device__ __forceinline__ void ssd_meet(float (&y)[4], int r) {
  if (RS >= 4) {             // lanes 2 apart trade halves, neighbours trade one of two, then the lanes 4, 8, .. apart add up
    const bool hi2 = (r & 2) != 0, hi1 = (r & 1) != 0;
    const float a0 = hi2 ? y[0] : y[2], a1 = hi2 ? y[1] : y[3];
    const float b0 = __shfl_xor_sync(0xffffffffu, a0, 2), b1 = __shfl_xor_sync(0xffffffffu, a1, 2);
    const float k0 = (hi2 ? y[2] : y[0]) + b0, k1 = (hi2 ? y[3] : y[1]) + b1;
    const float b = __shfl_xor_sync(0xffffffffu, hi1 ? k0 : k1, 1);
    y[0] = (hi1 ? k1 : k0) + b;
#pragma unroll
    for (int o = 4; o < RS; o <<= 1) y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
  } else if (RS == 2) {
    const bool hi = (r & 1) != 0;
    const float a0 = hi ? y[0] : y[2], a1 = hi ? y[1] : y[3];
    const float b0 = __shfl_xor_sync(0xffffffffu, a0, 1), b1 = __shfl_xor_sync(0xffffffffu, a1, 1);
    y[0] = (hi ? y[2] : y[0]) + b0;
    y[1] = (hi ? y[3] : y[1]) + b1;
  }
}

// Two fp32 numbers in a 64-bit register: one instruction multiplies or multiplies-and-adds both (each rounded like its
// scalar form).
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(lo), "f"(hi));
  return v;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
  float2 o;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(o.x), "=f"(o.y) : "l"(v));
  return o;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}

// one thread's share of a head's state: S[j][k] holds rows ssd_row(j / 2, r) + 2 (j % 2) and the next, column k
template <int RS>
__device__ __forceinline__ int ssd_row(int i, int r) { return 4 * (i * RS + r); }

__device__ __forceinline__ float4 ssd_load4(const float* p, int left, bool vec) {
  if (vec) return *reinterpret_cast<const float4*>(p);
  return make_float4(p[0], left > 1 ? p[1] : 0.f, left > 2 ? p[2] : 0.f, left > 3 ? p[3] : 0.f);
}
__device__ __forceinline__ void ssd_store4(float* p, float4 v, int left, bool vec) {
  if (vec) {
    *reinterpret_cast<float4*>(p) = v;
    return;
  }
  p[0] = v.x;
  if (left > 1) p[1] = v.y;
  if (left > 2) p[2] = v.z;
  if (left > 3) p[3] = v.w;
}

template <int RS>
__device__ __forceinline__ void ssd_load_state(f32x2 (&S)[8][4], const float* st, int N, int P, int e, int r, bool vec) {
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int n = ssd_row<RS>(j / 2, r) + 2 * (j % 2);
    const float* p = st + (size_t)n * P + e;
    const float4 a = (n < N && e < P) ? ssd_load4(p, P - e, vec) : zero;
    const float4 b = (n + 1 < N && e < P) ? ssd_load4(p + P, P - e, vec) : zero;
    S[j][0] = pack2(a.x, b.x); S[j][1] = pack2(a.y, b.y); S[j][2] = pack2(a.z, b.z); S[j][3] = pack2(a.w, b.w);
  }
}

template <int RS>
__device__ __forceinline__ void ssd_store_state(const f32x2 (&S)[8][4], float* st, int N, int P, int e, int r, bool vec) {
  if (e >= P) return;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int n = ssd_row<RS>(j / 2, r) + 2 * (j % 2);
    float* p = st + (size_t)n * P + e;
    const float2 x = unpack2(S[j][0]), y = unpack2(S[j][1]), z = unpack2(S[j][2]), w = unpack2(S[j][3]);
    if (n < N) ssd_store4(p, make_float4(x.x, y.x, z.x, w.x), P - e, vec);
    if (n + 1 < N) ssd_store4(p + P, make_float4(x.y, y.y, z.y, w.y), P - e, vec);
  }
}

// one token: S <- f S + B v^T (v = d x), and with OUT the thread's part of S^T C
template <int RS, bool OUT>
__device__ __forceinline__ void ssd_token(f32x2 (&S)[8][4], const float* B, const float* C, float f, float4 v, int r,
                                          float (&y)[4]) {
  const f32x2 ff = pack2(f, f);
  const f32x2 vv[4] = {pack2(v.x, v.x), pack2(v.y, v.y), pack2(v.z, v.z), pack2(v.w, v.w)};
  f32x2 acc[4] = {0ull, 0ull, 0ull, 0ull};                         // (two zeros)
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(B + ssd_row<RS>(i, r));
    ulonglong2 c = make_ulonglong2(0ull, 0ull);
    if (OUT) c = *reinterpret_cast<const ulonglong2*>(C + ssd_row<RS>(i, r));
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      S[2 * i][k] = fma2(ff, S[2 * i][k], mul2(b.x, vv[k]));
      if (OUT) acc[k] = fma2(S[2 * i][k], c.x, acc[k]);
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      S[2 * i + 1][k] = fma2(ff, S[2 * i + 1][k], mul2(b.y, vv[k]));
      if (OUT) acc[k] = fma2(S[2 * i + 1][k], c.y, acc[k]);
    }
  }
  if (OUT) {
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 a = unpack2(acc[k]);
      y[k] = a.x + a.y;
    }
  }
}

// y of a token written by the lanes that hold the sums; `x` are the token's value columns from e on (D x joins here)
template <int RS>
__device__ __forceinline__ void ssd_write(const float (&y)[4], const float* x, float D, float* out, int e, int P, int r) {
  constexpr int L = RS < 4 ? RS : 4, K = 4 / L;                    // lanes that write, columns of each
  if (r >= L) return;
#pragma unroll
  for (int k = 0; k < K; ++k) {
    const int c = r * K + k;
    if (e + c < P) out[e + c] = fmaf(D, x[c], y[k]);
  }
}

template <int RS> struct SsdTile {
  static constexpr int NPAD = 16 * RS;                             // rows, padded
  static constexpr int COLS = RS <= 8 ? 512 / RS : 64;             // columns of a block
  static constexpr int CH = RS <= 8 ? 8 : 4;                       // tokens fetched together
  static constexpr int ROW = 2 * NPAD + COLS + 4;                  // B | C | x | d, f
};

inline int ssd_row_split(int N) {
  int rs = 1;
  while (rs * 16 < N) rs *= 2;
  return rs;
}
template <int RS> inline dim3 ssd_block(int P) {
  const int cols = P < SsdTile<RS>::COLS ? P : SsdTile<RS>::COLS;
  const int threads = RS * ((cols + 3) / 4);
  return dim3((threads + 31) / 32 * 32);
}
template <int RS> inline int ssd_col_blocks(int P) { return (P + SsdTile<RS>::COLS - 1) / SsdTile<RS>::COLS; }

}  // namespace dlgo
