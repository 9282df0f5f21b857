// The recurrence with a decay per head (S_t = f_t S_(t-1) + d_t B_t x_t^T, y_t = S_t^T C_t + D x_t, S [N, P] per head) for
// prompts in bfloat16, on the tensor cores: B, C and x are bfloat16, everything else is fp32.
//
// With l_i the sum of the logarithms of f over a chunk's tokens up to i, a chunk of 64 tokens from the state S is
//   y_i = exp(l_i) S^T C_i + sum_(j <= i) (C_i . B_j) exp(l_i - l_j) d_j x_j + D x_i
//   S   <- exp(l_last) S + sum_j B_j (exp(l_last - l_j) d_j x_j)^T
// which are four matrix products (C B^T; C S; the masked C B^T times x; B^T times the scaled x).  A factor that is not
// bfloat16 by itself (the masked products, the scaled x, the state) enters as two bfloat16 terms, its rounding and what
// the rounding left, so that the sums keep about sixteen bits of it; all sums are fp32.  Only differences of l that are
// at most zero are raised, so strong decays neither overflow nor divide.
//
// A sequence's tokens are cut into segments that run side by side (LOCAL: the end every segment but the last reaches
// from zero; carry, see ssd.cuh; FULL: outputs from the carried starts).  A block owns (segment, head, 64 columns of x);
// a warp owns 16 of those columns for all tokens and keeps its part of the state, transposed, in the accumulators of the
// state's product, whose register layout is that of the second operand of C S.  Products are warp-level
// (mma.sync m16n8k16): each is a few thousand multiplications between element-wise passes over the accumulators, which
// stay in registers.
//
// With a normalizer (matrix memory) the recurrence also runs on x = 1: n_t = f_t n_(t-1) + d_t B_t, and n_t . C_t leaves
// per token and head.  Its chunk form needs the row sums of the masked products, which pass through registers anyway;
// the blocks of a head's first 64 columns carry it.
#include "ssd.cuh"

namespace dlgo {

constexpr int TC_TOKENS = 64, TC_COLS = 64, TC_PAD = 8;      // tokens of a chunk, columns of a block, elements between rows

__device__ __forceinline__ void mma_bf16(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// four 8 x 8 matrices of 16-bit numbers; lane i gives the address of row i % 8 of matrix i / 8
__device__ __forceinline__ void ldsm4(unsigned (&r)[4], const __nv_bfloat16* p) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ldsm4_t(unsigned (&r)[4], const __nv_bfloat16* p) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
// 16 bytes to shared memory, or 16 zero bytes
__device__ __forceinline__ void copy16_or_zero(__nv_bfloat16* dst, const __nv_bfloat16* src, bool in) {
  const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ unsigned bits(__nv_bfloat162 v) { return *reinterpret_cast<unsigned*>(&v); }
// (a, b) as two bfloat16 pairs: the rounding, and the rounding of what it left
__device__ __forceinline__ void split2(float a, float b, unsigned& hi, unsigned& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  hi = bits(h);
  lo = bits(__floats2bfloat162_rn(a - f.x, b - f.y));
}

struct SsdChunkArgs {
  const __nv_bfloat16* xbc;       // [T, ld]
  int ld, x0, b0, c0;             // columns of head 0's x, group 0's B and C
  const float* steps;             // [T, H, 2]: d, logarithm of f; null: d = 1, log_decay
  const float* log_decay;         // [H]
  const float* D;                 // [H] or null
  const int* tiles;
  int n_tiles;
  const int* seq_slot;
  float* state;
  long long state_ld;
  float* seg;                     // [n_tiles, H, N, P]
  float* seg_decay;               // [n_tiles, H]
  float* out;                     // [T, ldo]
  int ldo, direct;
  SsdShape s;
  float* norm_state;              // [slots at state_ld][H, N]: the normalizer's state, or null: none
  float* norm_seg;                // [n_tiles, H, N]
  float* norm_out;                // [T, H]: n_t . C_t
};

enum { CHUNK_LOCAL = 0, CHUNK_FULL = 1 };

template <int NT> struct SsdChunk {
  static constexpr int N = 16 * NT, LDN = N + TC_PAD, LDX = TC_COLS + TC_PAD, LDM = TC_TOKENS + TC_PAD;
  static constexpr int HALVES = 2 * TC_TOKENS * LDN + TC_TOKENS * LDX + 2 * TC_TOKENS * LDM;    // C, B, x, M (two terms)
  static constexpr size_t BYTES = sizeof(__nv_bfloat16) * HALVES + sizeof(float) * (4 * TC_TOKENS + N);
};

template <int NT, int MODE>
__global__ void __launch_bounds__(128, NT <= 4 ? 4 : 3)
ssd_chunks_kernel(SsdChunkArgs a) {
  using SC = SsdChunk<NT>;
  constexpr int LDN = SC::LDN, LDX = SC::LDX, LDM = SC::LDM;
  pdl_launch_dependents();
  extern __shared__ __align__(16) unsigned char smem[];
  __nv_bfloat16* Cs = reinterpret_cast<__nv_bfloat16*>(smem);      // [64][LDN]
  __nv_bfloat16* Bs = Cs + TC_TOKENS * LDN;                        // [64][LDN]
  __nv_bfloat16* Xs = Bs + TC_TOKENS * LDN;                        // [64][LDX]
  __nv_bfloat16* Mh = Xs + TC_TOKENS * LDX;                        // [64][LDM]
  __nv_bfloat16* Ml = Mh + TC_TOKENS * LDM;
  float* ls = reinterpret_cast<float*>(Ml + TC_TOKENS * LDM);      // [64] running sums of the logarithms
  float* ds = ls + TC_TOKENS;                                      // [64] d
  float* ws = ds + TC_TOKENS;                                      // [64] exp(l_last - l_j) d_j
  float* rsum = ws + TC_TOKENS;                                    // [64] row sums of the masked products (normalizer)
  float* ns = rsum + TC_TOKENS;                                    // [N] the normalizer
  const SsdShape& s = a.s;
  const int tile = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * TC_COLS;
  const int seq = a.tiles[tile * 3 + 0], t0 = a.tiles[tile * 3 + 1], count = a.tiles[tile * 3 + 2];
  const bool last = tile + 1 == a.n_tiles || a.tiles[(tile + 1) * 3] != seq;
  if (MODE == CHUNK_LOCAL && last) return;                         // nobody starts from its end
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n_warps = blockDim.x >> 5;
  const int N = s.N, P = s.P, g = h / (s.H / s.G), nx = min(TC_COLS, P - e0);
  const int r = lane >> 2, c2 = (lane & 3) * 2;                    // an accumulator's row and first column
  const int mrow = (lane & 7) + ((lane >> 3) & 1) * 8, mcol = (lane >> 4) * 8;   // ldmatrix: rows 0-15, then columns 8-15
  const int nrow = (lane & 7) + (lane >> 4) * 8, ncol = ((lane >> 3) & 1) * 8;   // ldmatrix: columns 0-15, then rows 8-15
  const float Dh = a.D != nullptr ? a.D[h] : 0.f;
  const float ldec = a.log_decay != nullptr ? a.log_decay[h] : 0.f;
  float* st = a.state + (size_t)a.seq_slot[seq] * a.state_ld + (size_t)h * N * P;
  float* sg = a.seg != nullptr ? a.seg + ((size_t)tile * s.H + h) * N * P : nullptr;
  const __nv_bfloat16* xg = a.xbc + a.x0 + (size_t)h * P + e0;
  const __nv_bfloat16* bg = a.xbc + a.b0 + (size_t)g * N;
  const __nv_bfloat16* cg = a.xbc + a.c0 + (size_t)g * N;
  pdl_wait();
  // S[t][.]: the state, transposed: columns p = warp * 16 + r (and + 8), rows n = 8 t + c2 (and + 1)
  float S[2 * NT][4];
  const int p0 = e0 + warp * 16 + r;
  {
    const float* src = a.direct ? st : sg;
#pragma unroll
    for (int t = 0; t < 2 * NT; ++t)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int n = 8 * t + c2 + (q & 1), p = p0 + (q >> 1) * 8;
        S[t][q] = (MODE == CHUNK_FULL && n < N && p < P) ? src[(size_t)n * P + p] : 0.f;
      }
  }
  const bool norm = a.norm_out != nullptr && blockIdx.z == 0;
  float* nst = norm ? a.norm_state + (size_t)a.seq_slot[seq] * a.state_ld + (size_t)h * N : nullptr;
  float* nsg = norm && a.norm_seg != nullptr ? a.norm_seg + ((size_t)tile * s.H + h) * N : nullptr;
  if (norm)
    for (int n = tid; n < SC::N; n += blockDim.x)
      ns[n] = (MODE == CHUNK_FULL && n < N) ? (a.direct ? nst : nsg)[n] : 0.f;
  float total_log = 0.f;
  for (int b = 0; b < count; b += TC_TOKENS) {
    const int nt = min(TC_TOKENS, count - b), tok0 = t0 + b;
    __syncthreads();                                               // the chunk before has been read
    for (int i = tid; i < TC_TOKENS * (2 * NT); i += blockDim.x) {
      const int t = i / (2 * NT), p = (i - t * (2 * NT)) * 8;
      const bool in = t < nt && p < N;
      const size_t row = (size_t)(tok0 + (in ? t : 0)) * a.ld + (in ? p : 0);
      copy16_or_zero(Bs + t * LDN + p, bg + row, in);
      if (MODE == CHUNK_FULL) copy16_or_zero(Cs + t * LDN + p, cg + row, in);
    }
    for (int i = tid; i < TC_TOKENS * (TC_COLS / 8); i += blockDim.x) {
      const int t = i / (TC_COLS / 8), p = (i - t * (TC_COLS / 8)) * 8;
      const bool in = t < nt && p < nx;
      copy16_or_zero(Xs + t * LDX + p, xg + (size_t)(tok0 + (in ? t : 0)) * a.ld + (in ? p : 0), in);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (warp == 0) {
      // two tokens per lane: steps, and the running sum of the logarithms
      float d[2], l[2];
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const int t = 2 * lane + q;
        d[q] = 0.f;
        l[q] = 0.f;
        if (t < nt) {
          if (a.steps != nullptr) {
            const float2 v = *reinterpret_cast<const float2*>(a.steps + ((size_t)(tok0 + t) * s.H + h) * 2);
            d[q] = v.x;
            l[q] = v.y;
          } else {
            d[q] = 1.f;
            l[q] = ldec;
          }
        }
      }
      float sum = l[0] + l[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
      }
      const float all = __shfl_sync(0xffffffffu, sum, 31);
      const float l1 = sum, l0 = sum - l[1];
      ls[2 * lane] = l0;
      ls[2 * lane + 1] = l1;
      ds[2 * lane] = d[0];
      ds[2 * lane + 1] = d[1];
      ws[2 * lane] = expf(all - l0) * d[0];
      ws[2 * lane + 1] = expf(all - l1) * d[1];
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const float l_last = ls[TC_TOKENS - 1];
    if (MODE == CHUNK_FULL) {
      // M = (C B^T) exp(l_i - l_j) d_j for j <= i, 16 rows per warp and trip
      for (int mt = warp; mt < 4; mt += n_warps) {
        if (mt * 16 >= nt) break;
        unsigned ca[NT][4];
#pragma unroll
        for (int kt = 0; kt < NT; ++kt) ldsm4(ca[kt], Cs + (mt * 16 + mrow) * LDN + kt * 16 + mcol);
        const int i0 = mt * 16 + r;
        const float li0 = ls[i0], li1 = ls[i0 + 8];
        float sum0 = 0.f, sum1 = 0.f;                              // of rows i0 and i0 + 8
        for (int jt = 0; jt <= mt; ++jt) {
          float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}}, odd[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
          for (int kt = 0; kt < NT; ++kt) {        // (sums over even and odd steps: four chains of products in flight)
            unsigned bb[4];
            ldsm4(bb, Bs + (jt * 16 + nrow) * LDN + kt * 16 + ncol);
            mma_bf16(kt & 1 ? odd[0] : acc[0], ca[kt], bb[0], bb[1]);
            mma_bf16(kt & 1 ? odd[1] : acc[1], ca[kt], bb[2], bb[3]);
          }
#pragma unroll
          for (int q = 0; q < 2; ++q)
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[q][k] += odd[q][k];
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            const int j = jt * 16 + q * 8 + c2;
            const float2 lj = *reinterpret_cast<const float2*>(ls + j), dj = *reinterpret_cast<const float2*>(ds + j);
            unsigned hi, lo;
            const float m00 = j <= i0 ? acc[q][0] * expf(li0 - lj.x) * dj.x : 0.f;
            const float m01 = j + 1 <= i0 ? acc[q][1] * expf(li0 - lj.y) * dj.y : 0.f;
            split2(m00, m01, hi, lo);
            *reinterpret_cast<unsigned*>(Mh + i0 * LDM + j) = hi;
            *reinterpret_cast<unsigned*>(Ml + i0 * LDM + j) = lo;
            const float m10 = j <= i0 + 8 ? acc[q][2] * expf(li1 - lj.x) * dj.x : 0.f;
            const float m11 = j + 1 <= i0 + 8 ? acc[q][3] * expf(li1 - lj.y) * dj.y : 0.f;
            split2(m10, m11, hi, lo);
            *reinterpret_cast<unsigned*>(Mh + (i0 + 8) * LDM + j) = hi;
            *reinterpret_cast<unsigned*>(Ml + (i0 + 8) * LDM + j) = lo;
            sum0 += m00 + m01;
            sum1 += m10 + m11;
          }
        }
        if (norm) {
#pragma unroll
          for (int o = 1; o < 4; o <<= 1) {
            sum0 += __shfl_xor_sync(0xffffffffu, sum0, o);
            sum1 += __shfl_xor_sync(0xffffffffu, sum1, o);
          }
          if ((lane & 3) == 0) {
            rsum[i0] = sum0;
            rsum[i0 + 8] = sum1;
          }
        }
      }
      __syncthreads();
      if (norm) {
        // two lanes per token: the start's normalizer against the token's C, and the chunk's own tokens
        for (int i = tid >> 1; i < TC_TOKENS; i += blockDim.x >> 1) {
          const __nv_bfloat16* crow = Cs + i * LDN;
          float dot = 0.f;
          for (int n = (tid & 1) * 8; n < SC::N; n += 16) {
            const uint4 v = *reinterpret_cast<const uint4*>(crow + n);
            const unsigned w4[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int q = 0; q < 4; ++q) {
              const float2 c = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w4[q]));
              dot = fmaf(c.x, ns[n + 2 * q], fmaf(c.y, ns[n + 2 * q + 1], dot));
            }
          }
          dot += __shfl_xor_sync(0xffffffffu, dot, 1);
          if ((tid & 1) == 0 && i < nt) a.norm_out[(size_t)(tok0 + i) * s.H + h] = fmaf(expf(ls[i]), dot, rsum[i]);
        }
        __syncthreads();                                           // every token has read the normalizer
      }
      // y: what the chunk's start brings ...
      float y[4][2][4];
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int q = 0; q < 2; ++q)
#pragma unroll
          for (int k = 0; k < 4; ++k) y[mt][q][k] = 0.f;
#pragma unroll
      for (int kt = 0; kt < NT; ++kt) {
        unsigned sh[2][2], sl[2][2];                               // [columns 0-7, 8-15][rows 0-7, 8-15 of the 16]
#pragma unroll
        for (int q = 0; q < 2; ++q)
#pragma unroll
          for (int k = 0; k < 2; ++k) split2(S[2 * kt + k][2 * q], S[2 * kt + k][2 * q + 1], sh[q][k], sl[q][k]);
        unsigned ca[4][4];                                         // (rows beyond the chunk's tokens are zeros)
#pragma unroll
        for (int mt = 0; mt < 4; ++mt) ldsm4(ca[mt], Cs + (mt * 16 + mrow) * LDN + kt * 16 + mcol);
#pragma unroll
        for (int mt = 0; mt < 4; ++mt)
#pragma unroll
          for (int q = 0; q < 2; ++q) mma_bf16(y[mt][q], ca[mt], sh[q][0], sh[q][1]);
#pragma unroll
        for (int mt = 0; mt < 4; ++mt)
#pragma unroll
          for (int q = 0; q < 2; ++q) mma_bf16(y[mt][q], ca[mt], sl[q][0], sl[q][1]);
      }
#pragma unroll
      for (int mt = 0; mt < 4; ++mt) {
        const float f0 = expf(ls[mt * 16 + r]), f1 = expf(ls[mt * 16 + r + 8]);
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          y[mt][q][0] *= f0; y[mt][q][1] *= f0;
          y[mt][q][2] *= f1; y[mt][q][3] *= f1;
        }
      }
      // ... and the chunk's own tokens
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        if (kt * 16 >= nt) break;
        unsigned xb[4];                                            // columns 0-7: rows 0-7, 8-15; columns 8-15: the same
        ldsm4_t(xb, Xs + (kt * 16 + mrow) * LDX + warp * 16 + mcol);
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int mt = kt; mt < 4; ++mt) {
            if (mt * 16 >= nt) break;
            unsigned m[4];
            ldsm4(m, (term ? Ml : Mh) + (mt * 16 + mrow) * LDM + kt * 16 + mcol);
            mma_bf16(y[mt][0], m, xb[0], xb[1]);
            mma_bf16(y[mt][1], m, xb[2], xb[3]);
          }
      }
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          const int i = mt * 16 + r + k * 8;
          if (i >= nt) continue;
          float* dst = a.out + (size_t)(tok0 + i) * a.ldo + (size_t)h * P + e0;
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            const int p = warp * 16 + q * 8 + c2;
            if (p >= nx) continue;                                 // (P is a multiple of 8: pairs are whole)
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(Xs + i * LDX + p));
            *reinterpret_cast<float2*>(dst + p) = make_float2(fmaf(Dh, x.x, y[mt][q][2 * k]), fmaf(Dh, x.y, y[mt][q][2 * k + 1]));
          }
        }
    }
    // the state at the chunk's end
    if (MODE == CHUNK_FULL && !last && b + TC_TOKENS >= count) break;    // (nobody reads it)
    total_log += l_last;
    const float fl = expf(l_last);
    if (norm) {
      for (int n = tid; n < SC::N; n += blockDim.x) {
        float v = fl * ns[n];
#pragma unroll 8
        for (int j = 0; j < TC_TOKENS; ++j) v = fmaf(ws[j], __bfloat162float(Bs[j * LDN + n]), v);   // (zeros beyond the chunk)
        ns[n] = v;
      }
    }
#pragma unroll
    for (int t = 0; t < 2 * NT; ++t)
#pragma unroll
      for (int q = 0; q < 4; ++q) S[t][q] *= fl;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      if (kt * 16 >= nt) break;
      unsigned xt[4], xh[4], xl[4];                                // x^T: rows p, columns tokens
      ldsm4_t(xt, Xs + (kt * 16 + nrow) * LDX + warp * 16 + ncol);
      const float2 w0 = *reinterpret_cast<const float2*>(ws + kt * 16 + c2), w1 = *reinterpret_cast<const float2*>(ws + kt * 16 + 8 + c2);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 v = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&xt[q]));
        const float2 w = q < 2 ? w0 : w1;
        split2(v.x * w.x, v.y * w.y, xh[q], xl[q]);
      }
      constexpr int TB = NT < 4 ? NT : 4;                          // tiles of B in flight
#pragma unroll
      for (int tb = 0; tb < NT; tb += TB) {
        unsigned bb[TB][4];                                        // rows (tokens) 0-7, 8-15 of columns 0-7, then of 8-15
#pragma unroll
        for (int t = 0; t < TB; ++t) ldsm4_t(bb[t], Bs + (kt * 16 + mrow) * LDN + (tb + t) * 16 + mcol);
#pragma unroll
        for (int t = 0; t < TB; ++t) {
          mma_bf16(S[2 * (tb + t)], xh, bb[t][0], bb[t][1]);
          mma_bf16(S[2 * (tb + t) + 1], xh, bb[t][2], bb[t][3]);
        }
#pragma unroll
        for (int t = 0; t < TB; ++t) {
          mma_bf16(S[2 * (tb + t)], xl, bb[t][0], bb[t][1]);
          mma_bf16(S[2 * (tb + t) + 1], xl, bb[t][2], bb[t][3]);
        }
      }
    }
  }
  if (MODE == CHUNK_LOCAL || last) {
    float* dst = MODE == CHUNK_LOCAL ? sg : st;
#pragma unroll
    for (int t = 0; t < 2 * NT; ++t)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int n = 8 * t + c2 + (q & 1), p = p0 + (q >> 1) * 8;
        if (n < N && p < P) dst[(size_t)n * P + p] = S[t][q];
      }
    if (norm)
      for (int n = tid; n < N; n += blockDim.x) (MODE == CHUNK_LOCAL ? nsg : nst)[n] = ns[n];      // (the thread's own)
  }
  if (MODE == CHUNK_LOCAL && tid == 0 && blockIdx.z == 0) a.seg_decay[(size_t)tile * s.H + h] = expf(total_log);
}

template <int NT>
static int launch_ssd_chunks(const SsdChunkArgs& a, cudaStream_t stream) {
  const size_t smem = SsdChunk<NT>::BYTES;
  const int cols = a.s.P < TC_COLS ? a.s.P : TC_COLS;
  const dim3 grid(a.n_tiles, a.s.H, (a.s.P + TC_COLS - 1) / TC_COLS), block((cols + 15) / 16 * 32);
  if (smem > 48 * 1024) {
    cudaFuncSetAttribute(ssd_chunks_kernel<NT, CHUNK_LOCAL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    cudaFuncSetAttribute(ssd_chunks_kernel<NT, CHUNK_FULL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  }
  if (!a.direct) {
    launch_kernel(ssd_chunks_kernel<NT, CHUNK_LOCAL>, grid, block, smem, stream, a);
    int st = launch_status();
    if (st != DLGO_OK) return st;
    st = launch_ssd_carry(a.tiles, a.n_tiles, a.seq_slot, a.state, a.state_ld, a.seg, a.seg_decay, a.s, stream);
    if (st != DLGO_OK) return st;
    if (a.norm_out != nullptr) {                                   // the normalizer as a state of one column
      st = launch_ssd_carry(a.tiles, a.n_tiles, a.seq_slot, a.norm_state, a.state_ld, a.norm_seg, a.seg_decay,
                            SsdShape{a.s.H, a.s.G, a.s.N, 1, 1}, stream);
      if (st != DLGO_OK) return st;
    }
  }
  launch_kernel(ssd_chunks_kernel<NT, CHUNK_FULL>, grid, block, smem, stream, a);
  return launch_status();
}

}  // namespace dlgo

using namespace dlgo;

// 1 if the kernels take these sizes: up to 128 state rows, rows of B, C and x in whole 16-byte pieces
DLGO_EXPORT int dlgo_ssd_chunks_takes(int N, int P) { return N > 0 && N <= 128 && N % 8 == 0 && P > 0 && P % 8 == 0; }

// xbc [T, ld] bfloat16; columns x0 (H heads of P), b0 and c0 (G groups of N); steps [T, H, 2] fp32 (d, logarithm of f), or
// null: d = 1 and log_decay [H]; D [H] fp32 or null; tiles [n_tiles, 3], a sequence's segments side by side in token
// order; out [T, ldo >= H P] fp32.  `direct`: one segment per sequence; else scratch holds n_tiles * H * (N P + 1) floats.
// norm_out [T, H] fp32 or null: n_t . C_t of the recurrence on x = 1, whose state [H, N] lies at norm_state + slot *
// state_ld; scratch then holds n_tiles * H * N floats more.
DLGO_EXPORT int dlgo_ssd_chunks(const void* xbc, int ld, int x0, int b0, int c0, const float* steps, const float* log_decay,
                                const float* D, const int* tiles, int n_tiles, int direct, const int* seq_slot, float* state,
                                long long state_ld, float* scratch, float* out, int ldo, int H, int G, int N, int P,
                                float* norm_state, float* norm_out, cudaStream_t stream) {
  if (n_tiles <= 0) return DLGO_OK;
  if (H <= 0 || H > 65535 || G <= 0 || H % G || n_tiles > 65535 || !dlgo_ssd_chunks_takes(N, P) || (steps == nullptr) == (log_decay == nullptr) ||
      (!direct && scratch == nullptr) || (norm_out != nullptr && norm_state == nullptr))
    return DLGO_ERR_SIZE;
  if (((ld | x0 | b0 | c0) & 7) || ((uintptr_t)xbc & 15) || (ldo & 1) || ((uintptr_t)out & 7)) return DLGO_ERR_ALIGN;
  SsdChunkArgs a{(const __nv_bfloat16*)xbc, ld, x0, b0, c0, steps, log_decay, D, tiles, n_tiles, seq_slot, state, state_ld,
                 direct ? nullptr : scratch, direct ? nullptr : scratch + (size_t)n_tiles * H * N * P, out, ldo, direct,
                 SsdShape{H, G, N, P, 1}, norm_state,
                 direct || norm_out == nullptr ? nullptr : scratch + (size_t)n_tiles * H * (N * P + 1), norm_out};
  if (N <= 16) return launch_ssd_chunks<1>(a, stream);
  if (N <= 32) return launch_ssd_chunks<2>(a, stream);
  if (N <= 64) return launch_ssd_chunks<4>(a, stream);
  return launch_ssd_chunks<8>(a, stream);
}
