// The real-gated linear recurrent unit (Griffin) with its short convolution over time.  Per channel c of W, which lie in
// `parts` equal parts of B neighbours:
//
//   u_t = bc + sum_j taps[c, j] x_(t - n + 1 + j)             x = the projection's number plus bx; 0 before a sequence's start
//   r_t = sigmoid(zr + br),  i_t = sigmoid(zi + bi)           zr, zi: products of the channel's rows of two [B, B] matrices
//                                                             with its part of u_t
//   log a_t = -rate r_t softplus(lam),  a_t = exp(log a_t)
//   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t               S = 0 before a sequence's start
//   out_t = S_t gelu(y_t + by)                                y: a second projection (tanh form of gelu)
//
// A sequence's state row is [W numbers of S | taps x W inputs x]: the input of position p lies in entry p mod taps, one
// entry more than is read back, so that a step's new input never lies where the same step still reads an old one.
//
// rglru_conv   prompts: u for all tokens (fp32, and the operand of the gates' contraction in the run's type, in rows of a
//              part: [parts, T, B], sorted by part, or [T, parts, B])
// rglru_scan   prompts: a sequence's tokens are cut into segments that run side by side
//                LOCAL   a and the input of every token take the places of the gates' logits; every segment's end from
//                        zero and the product of its a (as the sum of logarithms).  In bfloat16 the gates' contraction
//                        does this in its epilogue (rglru_tc.cu).
//                carry   the start of every segment from the stored state and the ends before it
//                FULL    every segment walks its tokens again from its start; the last one of a sequence stores the state
//                        and the inputs that the next step reads back
//              with one segment per sequence DIRECT runs alone from the logits
// rglru_step   decoding: convolution, gates, recurrence and output of one token per sequence in one launch
// Everything is fp32 but the gates' operand and weights, and y where the contraction before has finished it in bfloat16.
#include "common.cuh"

namespace dlgo {

struct RglruShape {
  int W, parts, taps;
  float rate;
  __host__ __device__ int B() const { return W / parts; }
};

__device__ __forceinline__ float rg_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float rg_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float rg_gelu(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// (log a, factor of u): from the gates' finished logits and softplus(lam) times the rate
__device__ __forceinline__ void rg_factors(float zr, float zi, float rate_sp, float& log_a, float& in) {
  log_a = -rate_sp * rg_sigmoid(zr);
  in = sqrtf(-expm1f(2.0f * log_a)) * rg_sigmoid(zi);
}

// ------------------------------------------------------------------------------- convolution (prompts)
constexpr int RC_THREADS = 128;

// A thread owns W4 neighbouring channels (4, or 1) and walks its tile's tokens with the taps' reach in registers.
template <typename TO, int TAPS, int W4>
__global__ void __launch_bounds__(RC_THREADS)
rglru_conv_kernel(const float* x, int ldx, const float* __restrict__ bx, const float* __restrict__ w_taps,
                  const float* __restrict__ bc, const int* __restrict__ tiles, const int* __restrict__ token_seq,
                  const int* __restrict__ token_pos, const int* __restrict__ seq_slot, const float* state,
                  long long state_ld, float* u_out, TO* rows, int by_part, int T, RglruShape s) {
  pdl_launch_dependents();
  const int tile = blockIdx.x;
  const int seq = tiles[tile * 3 + 0], t0 = tiles[tile * 3 + 1], count = tiles[tile * 3 + 2];
  const int c = (blockIdx.y * RC_THREADS + threadIdx.x) * W4;
  if (c >= s.W) return;
  const int n = TAPS > 0 ? TAPS : s.taps, pos0 = token_pos[t0];
  int first = t0;                                  // the sequence's first token of this step, if within the taps' reach
  while (first > 0 && first > t0 - n + 1 && token_seq[first - 1] == seq) --first;
  const float* ring = state + (size_t)seq_slot[seq] * state_ld + s.W;
  const int B = s.B(), part = c / B;
  float bias_x[W4], bias_c[W4];
#pragma unroll
  for (int k = 0; k < W4; ++k) {
    bias_x[k] = bx[c + k];
    bias_c[k] = bc[c + k];
  }
  // the input `back` tokens before packed token tok
  auto input = [&](int tok, int back, float (&v)[W4]) {
    const int at = tok - back, p = pos0 + (tok - t0) - back;
#pragma unroll
    for (int k = 0; k < W4; ++k) {
      v[k] = 0.f;
      if (at >= first) v[k] = x[(size_t)at * ldx + c + k] + bias_x[k];
      else if (p >= 0) v[k] = ring[(size_t)(p % n) * s.W + c + k];
    }
  };
  auto emit = [&](int t, const float (&y)[W4]) {
    float* dst = u_out == nullptr ? nullptr : u_out + (size_t)t * s.W + c;
    TO* row = rows == nullptr ? nullptr
                              : rows + (by_part ? ((size_t)part * T + t) * B + (c - part * B) : (size_t)t * s.W + c);
    if (W4 == 4) {
      if (dst != nullptr) *reinterpret_cast<float4*>(dst) = make_float4(y[0], y[1 % W4], y[2 % W4], y[3 % W4]);
      if (row != nullptr) {
        if (sizeof(TO) == 2) {
          __nv_bfloat162 h[2] = {__floats2bfloat162_rn(y[0], y[1 % W4]), __floats2bfloat162_rn(y[2 % W4], y[3 % W4])};
          *reinterpret_cast<uint2*>(row) = *reinterpret_cast<uint2*>(h);
        } else {
          *reinterpret_cast<float4*>(row) = make_float4(y[0], y[1 % W4], y[2 % W4], y[3 % W4]);
        }
      }
    } else {
      if (dst != nullptr) dst[0] = y[0];
      if (row != nullptr) row[0] = from_float<TO>(y[0]);
    }
  };
  if (TAPS > 0) {
    constexpr int R = TAPS > 0 ? TAPS : 1, FLY = 8;
    float tap[R][W4], v[R][W4];
#pragma unroll
    for (int j = 0; j < R; ++j)
#pragma unroll
      for (int k = 0; k < W4; ++k) tap[j][k] = w_taps[(size_t)(c + k) * R + j];
    pdl_wait();
#pragma unroll
    for (int j = 0; j < R - 1; ++j) input(t0, R - 1 - j, v[j]);
    for (int tb = 0; tb < count; tb += FLY) {
      float in[FLY][W4];                           // several tokens' fetches in flight
#pragma unroll
      for (int q = 0; q < FLY; ++q) {
        const float* src = x + (size_t)(t0 + min(tb + q, count - 1)) * ldx + c;
        if (W4 == 4) {
          const float4 a = *reinterpret_cast<const float4*>(src);
          in[q][0] = a.x; in[q][1 % W4] = a.y; in[q][2 % W4] = a.z; in[q][3 % W4] = a.w;
        } else {
          in[q][0] = src[0];
        }
      }
#pragma unroll
      for (int q = 0; q < FLY; ++q) {
        if (tb + q >= count) break;
        float y[W4];
#pragma unroll
        for (int k = 0; k < W4; ++k) {
          v[R - 1][k] = in[q][k] + bias_x[k];
          float a = bias_c[k];
#pragma unroll
          for (int j = 0; j < R; ++j) a = fmaf(tap[j][k], v[j][k], a);
          y[k] = a;
#pragma unroll
          for (int j = 0; j < R - 1; ++j) v[j][k] = v[j + 1][k];
        }
        emit(t0 + tb + q, y);
      }
    }
  } else {
    pdl_wait();
    for (int t = t0; t < t0 + count; ++t) {
      // (a tile may be longer than the taps' reach: the walk back stops at the tile's own first token)
      float y[W4];
#pragma unroll
      for (int k = 0; k < W4; ++k) y[k] = bias_c[k];
      for (int j = 0; j < n; ++j) {
        float v[W4];
        input(t, n - 1 - j, v);
#pragma unroll
        for (int k = 0; k < W4; ++k) y[k] = fmaf(w_taps[(size_t)(c + k) * n + j], v[k], y[k]);
      }
      emit(t, y);
    }
  }
}

// ------------------------------------------------------------------------------- recurrence (prompts)
// The start of every segment.  A block takes 32 channels of a sequence and CY_WAYS * CY_FLY segments at a time: a warp
// composes CY_FLY neighbouring segments (each a map S -> f S + e) of its lanes' channels, the warps' maps meet in shared
// memory, and every warp walks its segments again from its start.
constexpr int CY_WAYS = 8, CY_FLY = 8;
__global__ void __launch_bounds__(CY_WAYS * 32)
rglru_carry_kernel(const int* __restrict__ tiles, int n_tiles, const int* __restrict__ seq_slot, const float* state,
                   long long state_ld, float* seg, int W) {
  pdl_launch_dependents();
  __shared__ float f_s[CY_WAYS][32], e_s[CY_WAYS][32];
  const int j0 = blockIdx.y, seq = tiles[j0 * 3], lane = threadIdx.x & 31, way = threadIdx.x >> 5;
  if (j0 > 0 && tiles[(j0 - 1) * 3] == seq) return;                // a block row per first segment of a sequence
  const int c = min(blockIdx.x * 32 + lane, W - 1);                // (lanes beyond the channels repeat the last one)
  int end = j0 + 1;
  while (end < n_tiles && tiles[end * 3] == seq) ++end;
  pdl_wait();
  float S = state[(size_t)seq_slot[seq] * state_ld + c];
  for (int base = j0; base < end; base += CY_WAYS * CY_FLY) {
    const int j = base + way * CY_FLY;
    float e[CY_FLY], f[CY_FLY];
#pragma unroll
    for (int q = 0; q < CY_FLY; ++q) {
      const float* sg = seg + (size_t)min(j + q, end - 1) * 3 * W + c;
      e[q] = sg[0];
      f[q] = sg[W];
    }
    float F = 1.f, E = 0.f;
#pragma unroll
    for (int q = 0; q < CY_FLY; ++q) {
      f[q] = expf(f[q]);
      if (j + q < end) {
        F *= f[q];
        E = fmaf(f[q], E, e[q]);
      }
    }
    f_s[way][lane] = F;
    e_s[way][lane] = E;
    __syncthreads();
    float mine = S;
    for (int w = 0; w < CY_WAYS; ++w) {
      if (w == way) mine = S;
      S = fmaf(f_s[w][lane], S, e_s[w][lane]);
    }
#pragma unroll
    for (int q = 0; q < CY_FLY; ++q) {
      if (j + q < end) {
        seg[((size_t)(j + q) * 3 + 2) * W + c] = mine;
        mine = fmaf(f[q], mine, e[q]);
      }
    }
    __syncthreads();                                               // the maps have been read
  }
}

enum { RG_LOCAL = 0, RG_FULL = 1, RG_DIRECT = 2 };
constexpr int RS_THREADS = 128, RS_FLY = 8;

struct RglruScan {
  float* z;                       // [T, parts, 2 B]: logits of r, then of i; LOCAL leaves (a, input) in their places
  const float* u;                 // [T, W]
  const float* br;                // [W]
  const float* bi;                // [W]
  const float* lam;               // [W]
  const float* y32;               // [T, ldy] fp32 without bias and gelu, or null
  const float* by;                // [W] (y32)
  const __nv_bfloat16* y16;       // [T, ldy] finished, or null
  int ldy;
  const float* x;                 // [T, ldx], bx [W]: the convolution's inputs (kept for the next step)
  int ldx;
  const float* bx;
  const int* tiles;
  int n_tiles;
  const int* token_seq;
  const int* token_pos;
  const int* seq_slot;
  float* state;
  long long state_ld;
  float* seg;                     // [n_tiles, 3, W]: end from zero, sum of the logarithms, start
  RglruShape s;
};

template <typename TO, int MODE>
__global__ void __launch_bounds__(RS_THREADS)
rglru_scan_kernel(RglruScan a, TO* out) {
  pdl_launch_dependents();
  const RglruShape s = a.s;
  const int tile = blockIdx.x;
  const int seq = a.tiles[tile * 3 + 0], t0 = a.tiles[tile * 3 + 1], count = a.tiles[tile * 3 + 2];
  const int c = blockIdx.y * RS_THREADS + threadIdx.x;
  if (c >= s.W) return;
  const bool last = tile + 1 == a.n_tiles || a.tiles[(tile + 1) * 3] != seq;
  const int B = s.B(), part = c / B;
  const float b_r = a.br[c], b_i = a.bi[c], rate_sp = s.rate * rg_softplus(a.lam[c]);
  const float b_y = a.y32 != nullptr && MODE != RG_LOCAL ? a.by[c] : 0.f;
  float* row = a.state + (size_t)a.seq_slot[seq] * a.state_ld;
  float* z = a.z + (size_t)part * 2 * B + (c - part * B);
  const size_t ldz = (size_t)2 * s.W;
  pdl_wait();
  float S = 0.f;
  if (MODE == RG_DIRECT) S = row[c];
  if (MODE == RG_FULL) S = a.seg[((size_t)tile * 3 + 2) * s.W + c];    // (the stored state is replaced in this launch)
  float total = 0.f;
  for (int tb = 0; tb < count; tb += RS_FLY) {
    float f0[RS_FLY], f1[RS_FLY], uu[RS_FLY], yy[RS_FLY];
#pragma unroll
    for (int q = 0; q < RS_FLY; ++q) {
      const size_t t = (size_t)(t0 + min(tb + q, count - 1));
      f0[q] = z[t * ldz];
      f1[q] = z[t * ldz + B];
      uu[q] = MODE != RG_FULL ? a.u[t * s.W + c] : 0.f;
      yy[q] = 0.f;
      if (MODE != RG_LOCAL) yy[q] = a.y32 != nullptr ? a.y32[t * a.ldy + c] : __bfloat162float(a.y16[t * a.ldy + c]);
    }
#pragma unroll
    for (int q = 0; q < RS_FLY; ++q) {
      if (tb + q >= count) break;
      const size_t t = (size_t)(t0 + tb + q);
      float decay = f0[q], in = f1[q];
      if (MODE != RG_FULL) {
        float log_a, g;
        rg_factors(f0[q] + b_r, f1[q] + b_i, rate_sp, log_a, g);
        decay = expf(log_a);
        in = g * uu[q];
        if (MODE == RG_LOCAL) {
          total += log_a;
          z[t * ldz] = decay;
          z[t * ldz + B] = in;
        }
      }
      S = fmaf(decay, S, in);
      if (MODE != RG_LOCAL) {
        const float y = a.y32 != nullptr ? rg_gelu(yy[q] + b_y) : yy[q];
        out[t * s.W + c] = from_float<TO>(S * y);
      }
    }
  }
  if (MODE == RG_LOCAL) {
    float* sg = a.seg + (size_t)tile * 3 * s.W + c;
    sg[0] = S;
    sg[s.W] = total;
    return;
  }
  if (!last) return;
  row[c] = S;
  // the newest inputs, as many as there are entries and as this step brought (every reader of the old ones ran in an
  // earlier launch)
  const int end = t0 + count, pe = a.token_pos[end - 1];
  const float b_x = a.bx[c];
  for (int j = 0; j < s.taps; ++j) {
    const int t = end - 1 - j;
    if (t < 0 || a.token_seq[t] != seq) break;
    row[s.W + (size_t)((pe - j) % s.taps) * s.W + c] = a.x[(size_t)t * a.ldx + c] + b_x;
  }
}

// ------------------------------------------------------------------------------- one token per sequence
// A block owns CH neighbouring channels of one part for up to TOK tokens: their part of u in shared memory (a thread per
// channel, all inputs of all tokens in flight together), a warp per output channel at a time over the rows of both
// matrices, then the recurrence.
constexpr int ST_THREADS = 256, ST_CH = 16, ST_TOK = 8, ST_TAPS = 4;
static_assert(ST_CH * ST_TOK <= ST_THREADS, "the last pass has a thread per channel and token");

template <typename TW, int VEC> struct WRow;
template <typename TW> struct WRow<TW, 1> {
  static __device__ __forceinline__ void load(const TW* p, float (&o)[1]) { o[0] = to_float(p[0]); }
};
template <> struct WRow<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&o)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
  }
};
template <> struct WRow<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&o)[4]) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    o[0] = a.x; o[1] = a.y; o[2] = b.x; o[3] = b.y;
  }
};

// v[k] summed over the warp for k < 16: lane l ends with the sum of entry l >> 1 (halves of the entries are traded at
// distances 16, 8, 4, 2, then neighbours add up)
__device__ __forceinline__ float warp_sum16(float (&v)[16], int lane) {
#pragma unroll
  for (int o = 16, n = 8; n > 0; o >>= 1, n >>= 1) {
    const bool hi = (lane & o) != 0;
#pragma unroll
    for (int k = 0; k < n; ++k) {
      const float give = hi ? v[k] : v[k + n], keep = hi ? v[k + n] : v[k];
      v[k] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
  return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 1);
}

template <typename TW, typename TO, int VEC>
__global__ void __launch_bounds__(ST_THREADS, 2)
rglru_step_kernel(const float* proj, int ld, int x0, const float* __restrict__ by, const float* __restrict__ bx,
                  const float* __restrict__ w_taps, const float* __restrict__ bc, const TW* __restrict__ w_gates,
                  const float* __restrict__ br, const float* __restrict__ bi, const float* __restrict__ lam,
                  const int* __restrict__ token_pos, const int* __restrict__ seq_slot, float* state, long long state_ld,
                  TO* out, int T, int tok, RglruShape s) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float u_s[];                     // [tok][B]
  __shared__ float z_s[2][ST_TOK][ST_CH];
  __shared__ int pos_s[ST_TOK], entry_s[ST_TAPS - 1][ST_TOK];
  __shared__ long long row_s[ST_TOK];
  const int B = s.B(), n = s.taps, per_part = (B + ST_CH - 1) / ST_CH;
  const int part = blockIdx.x / per_part, o0 = (blockIdx.x - part * per_part) * ST_CH, no = min(ST_CH, B - o0);
  const int t0 = blockIdx.y * tok, nt = min(tok, T - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // this block's rows of the gates' weights: on their way before the wait
  for (int o = warp; o < 2 * no; o += ST_THREADS / 32) {
    const char* p = (const char*)(w_gates + ((size_t)part * 2 * B + (o & 1) * B + o0 + (o >> 1)) * B);
    for (int b = lane * 128; b < B * (int)sizeof(TW); b += 32 * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(p + b));
  }
  if (threadIdx.x < ST_TOK) {                                      // the step's own inputs (tokens beyond the last repeat it)
    const int t = t0 + min((int)threadIdx.x, nt - 1), pos = token_pos[t];
    pos_s[threadIdx.x] = pos;
    row_s[threadIdx.x] = (long long)seq_slot[t] * state_ld;
#pragma unroll
    for (int j = 0; j < ST_TAPS - 1; ++j) {                        // the entry of the input j + 1 tokens before, or none
      const int p = pos - 1 - j;
      entry_s[j][threadIdx.x] = (j < n - 1 && p >= 0) ? p % n : -1;
    }
  }
  __syncthreads();
  const int fq = threadIdx.x / ST_CH, fo = threadIdx.x - fq * ST_CH, fc = part * B + o0 + min(fo, no - 1);
  const bool fin = fq < nt && fo < no;
  float f_br = 0.f, f_bi = 0.f, f_rate = 0.f, f_by = 0.f, f_bx = 0.f;
  if (fin) {                                                       // weights
    f_br = br[fc];
    f_bi = bi[fc];
    f_rate = s.rate * rg_softplus(lam[fc]);
    f_by = by[fc];
    f_bx = bx[fc];
  }
  pdl_wait();
  // what the last pass needs of this block's own channels: requested now
  float S_old = 0.f, y_now = 0.f, x_now = 0.f;
  if (fin) {
    const float* pr = proj + (size_t)(t0 + fq) * ld;
    S_old = state[row_s[fq] + fc];
    y_now = pr[fc];
    x_now = pr[x0 + fc];
  }
  for (int i = threadIdx.x; i < B; i += ST_THREADS) {
    const int c = part * B + i;
    float now[ST_TOK], old[ST_TAPS - 1][ST_TOK], w[ST_TAPS - 1];
#pragma unroll
    for (int q = 0; q < ST_TOK; ++q) now[q] = proj[(size_t)(t0 + min(q, nt - 1)) * ld + x0 + c];
#pragma unroll
    for (int j = 0; j < ST_TAPS - 1; ++j) {
      w[j] = j < n - 1 ? w_taps[(size_t)c * n + n - 2 - j] : 0.f;
#pragma unroll
      for (int q = 0; q < ST_TOK; ++q) {
        const int entry = entry_s[j][q];
        old[j][q] = 0.f;
        if (entry >= 0) old[j][q] = state[row_s[q] + s.W + (size_t)entry * s.W + c];
      }
    }
    const float w_now = w_taps[(size_t)c * n + n - 1], b_x = bx[c], b_c = bc[c];
#pragma unroll
    for (int q = 0; q < ST_TOK; ++q) {
      float a = b_c;
      for (int j = n - 2; j >= ST_TAPS - 1; --j) {                 // taps beyond those in registers, oldest first
        const int p = pos_s[q] - 1 - j;
        if (p >= 0) a = fmaf(w_taps[(size_t)c * n + n - 2 - j], state[row_s[q] + s.W + (size_t)(p % n) * s.W + c], a);
      }
#pragma unroll
      for (int j = ST_TAPS - 2; j >= 0; --j) a = fmaf(w[j], old[j][q], a);
      a = fmaf(w_now, now[q] + b_x, a);
      if (q < nt) u_s[q * B + i] = a;
    }
  }
  __syncthreads();
  for (int o = warp; o < no; o += ST_THREADS / 32) {
    const TW* wr = w_gates + ((size_t)part * 2 * B + o0 + o) * B;
    const TW* wi = wr + (size_t)B * B;
    float acc[2 * ST_TOK];                                         // r of every token, then i
#pragma unroll
    for (int q = 0; q < 2 * ST_TOK; ++q) acc[q] = 0.f;
#pragma unroll 2
    for (int k = lane * VEC; k < B; k += 32 * VEC) {
      float r[VEC], i[VEC];
      WRow<TW, VEC>::load(wr + k, r);
      WRow<TW, VEC>::load(wi + k, i);
#pragma unroll
      for (int q = 0; q < ST_TOK; ++q) {
        if (q < nt) {
          float u[VEC];
          WRow<float, VEC>::load(u_s + q * B + k, u);
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            acc[q] = fmaf(r[e], u[e], acc[q]);
            acc[ST_TOK + q] = fmaf(i[e], u[e], acc[ST_TOK + q]);
          }
        }
      }
    }
    const float sum = warp_sum16(acc, lane);
    if ((lane & 1) == 0) z_s[lane >> 4][(lane >> 1) & (ST_TOK - 1)][o] = sum;
  }
  __syncthreads();
  if (fin) {
    float* row = state + row_s[fq];
    float log_a, g;
    rg_factors(z_s[0][fq][fo] + f_br, z_s[1][fq][fo] + f_bi, f_rate, log_a, g);
    const float S = fmaf(expf(log_a), S_old, g * u_s[fq * B + o0 + fo]);
    row[fc] = S;
    // (the entry of this position: no block of this launch reads it)
    row[s.W + (size_t)(pos_s[fq] % n) * s.W + fc] = x_now + f_bx;
    out[(size_t)(t0 + fq) * s.W + fc] = from_float<TO>(S * rg_gelu(y_now + f_by));
  }
}

static bool rglru_ok(const RglruShape& s) {
  return s.W > 0 && s.parts > 0 && s.W % s.parts == 0 && s.taps > 0 && s.rate > 0.f;
}

template <typename TO>
static int launch_rglru_conv(const float* x, int ldx, const float* bx, const float* w_taps, const float* bc, const int* tiles,
                             int n_tiles, const int* token_seq, const int* token_pos, const int* seq_slot, const float* state,
                             long long state_ld, float* u, TO* rows, int by_part, int T, const RglruShape& s,
                             cudaStream_t stream) {
  const bool four = s.taps >= 2 && s.taps <= 4 && ((s.B() | ldx) & 3) == 0 && (((uintptr_t)x | (uintptr_t)u | (uintptr_t)rows) & 15) == 0;
  const int w = four ? 4 : 1;
  const dim3 grid(n_tiles, (s.W + RC_THREADS * w - 1) / (RC_THREADS * w)), block(RC_THREADS);
#define RC_ARGS grid, block, 0, stream, x, ldx, bx, w_taps, bc, tiles, token_seq, token_pos, seq_slot, state, state_ld, u, rows, \
                by_part, T, s
  if (four && s.taps == 4) launch_kernel(rglru_conv_kernel<TO, 4, 4>, RC_ARGS);
  else if (four && s.taps == 3) launch_kernel(rglru_conv_kernel<TO, 3, 4>, RC_ARGS);
  else if (four && s.taps == 2) launch_kernel(rglru_conv_kernel<TO, 2, 4>, RC_ARGS);
  else launch_kernel(rglru_conv_kernel<TO, 0, 1>, RC_ARGS);
#undef RC_ARGS
  return launch_status();
}

template <typename TO>
static int launch_rglru_scan(const RglruScan& a, TO* out, int direct, int prepared, cudaStream_t stream) {
  const dim3 grid(a.n_tiles, (a.s.W + RS_THREADS - 1) / RS_THREADS), block(RS_THREADS);
  if (direct) {
    launch_kernel(rglru_scan_kernel<TO, RG_DIRECT>, grid, block, 0, stream, a, out);
    return launch_status();
  }
  int st = DLGO_OK;
  if (!prepared) {
    launch_kernel(rglru_scan_kernel<TO, RG_LOCAL>, grid, block, 0, stream, a, out);
    st = launch_status();
    if (st != DLGO_OK) return st;
  }
  launch_kernel(rglru_carry_kernel, dim3((a.s.W + 31) / 32, a.n_tiles), dim3(CY_WAYS * 32), 0, stream, a.tiles,
                a.n_tiles, a.seq_slot, (const float*)a.state, a.state_ld, a.seg, a.s.W);
  st = launch_status();
  if (st != DLGO_OK) return st;
  launch_kernel(rglru_scan_kernel<TO, RG_FULL>, grid, block, 0, stream, a, out);
  return launch_status();
}

template <typename TW, typename TO>
static int launch_rglru_step(const float* proj, int ld, int x0, const float* by, const float* bx, const float* w_taps,
                             const float* bc, const TW* w_gates, const float* br, const float* bi, const float* lam,
                             const int* token_pos, const int* seq_slot, float* state, long long state_ld, TO* out, int T,
                             const RglruShape& s, cudaStream_t stream) {
  const int B = s.B();
  int tok = ST_TOK;
  while (tok > 1 && (size_t)tok * B * sizeof(float) > 40 * 1024) tok >>= 1;
  const size_t smem = (size_t)tok * B * sizeof(float);
  if (smem > 200 * 1024) return DLGO_ERR_SIZE;
  const long long gx = (long long)s.parts * ((B + ST_CH - 1) / ST_CH);
  const dim3 grid((unsigned)gx, (T + tok - 1) / tok), block(ST_THREADS);
  const bool four = B % 4 == 0 && ((uintptr_t)w_gates & 15) == 0;
#define ST_ARGS grid, block, smem, stream, proj, ld, x0, by, bx, w_taps, bc, w_gates, br, bi, lam, token_pos, seq_slot, state, \
                state_ld, out, T, tok, s
  if (four) {
    if (smem > 40 * 1024) cudaFuncSetAttribute(rglru_step_kernel<TW, TO, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_kernel(rglru_step_kernel<TW, TO, 4>, ST_ARGS);
  } else {
    if (smem > 40 * 1024) cudaFuncSetAttribute(rglru_step_kernel<TW, TO, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_kernel(rglru_step_kernel<TW, TO, 1>, ST_ARGS);
  }
#undef ST_ARGS
  return launch_status();
}

}  // namespace dlgo

using namespace dlgo;

// x [T, ldx] fp32 (W columns), bx, bc [W], w_taps [W, taps] fp32; tiles [n_tiles, 3] (sequence, first packed token,
// count); u [T, W] fp32 or null; rows in `rows_dtype` or null: u as rows of a part, [parts, T, B] (by_part) or [T, W].
DLGO_EXPORT int dlgo_rglru_conv(const float* x, int ldx, const float* bx, const float* w_taps, const float* bc,
                                const int* tiles, int n_tiles, const int* token_seq, const int* token_pos,
                                const int* seq_slot, const float* state, long long state_ld, float* u, void* rows,
                                int rows_dtype, int by_part, int T, int W, int parts, int taps, cudaStream_t stream) {
  if (n_tiles <= 0 || T <= 0) return DLGO_OK;
  const RglruShape s{W, parts, taps, 1.f};
  if (!rglru_ok(s)) return DLGO_ERR_SIZE;
#define RC_CALL(T_) launch_rglru_conv<T_>(x, ldx, bx, w_taps, bc, tiles, n_tiles, token_seq, token_pos, seq_slot, state, state_ld, \
                                          u, (T_*)rows, by_part, T, s, stream)
  if (rows_dtype == DLGO_F32) return RC_CALL(float);
  if (rows_dtype == DLGO_BF16) return RC_CALL(__nv_bfloat16);
#undef RC_CALL
  return DLGO_ERR_DTYPE;
}

// z [T, parts, 2 B] fp32: the gates' logits without biases (r, then i); u of dlgo_rglru_conv; y: fp32 without bias and
// gelu (y_dtype 0, by [W]) or finished bfloat16 (y_dtype 1), row stride ldy; x, bx as in dlgo_rglru_conv; tiles: a
// sequence's segments side by side in token order; seg: n_tiles * 3 * W floats of scratch (unused when `direct`: one
// segment per sequence); out [T, W] in out_dtype.  `prepared` (not direct): z and seg hold what LOCAL leaves.
DLGO_EXPORT int dlgo_rglru_scan(float* z, const float* u, const float* br, const float* bi, const float* lam, const void* y,
                                int y_dtype, int ldy, const float* by, const float* x, int ldx, const float* bx,
                                const int* tiles, int n_tiles, const int* token_seq, const int* token_pos,
                                const int* seq_slot, float* state, long long state_ld, float* seg, int direct, int prepared,
                                void* out, int out_dtype, int W, int parts, int taps, float rate, cudaStream_t stream) {
  if (n_tiles <= 0) return DLGO_OK;
  const RglruShape s{W, parts, taps, rate};
  if (!rglru_ok(s) || (!direct && seg == nullptr) || (direct && prepared) || n_tiles > 65535 || (y_dtype == DLGO_F32 && by == nullptr)) return DLGO_ERR_SIZE;
  if (y_dtype != DLGO_F32 && y_dtype != DLGO_BF16) return DLGO_ERR_DTYPE;
  RglruScan a{z, u, br, bi, lam, y_dtype == DLGO_F32 ? (const float*)y : nullptr, by,
              y_dtype == DLGO_BF16 ? (const __nv_bfloat16*)y : nullptr, ldy, x, ldx, bx, tiles, n_tiles, token_seq,
              token_pos, seq_slot, state, state_ld, seg, s};
  if (out_dtype == DLGO_F32) return launch_rglru_scan<float>(a, (float*)out, direct, prepared, stream);
  if (out_dtype == DLGO_BF16) return launch_rglru_scan<__nv_bfloat16>(a, (__nv_bfloat16*)out, direct, prepared, stream);
  return DLGO_ERR_DTYPE;
}

// One token per sequence (token t belongs to sequence t).  proj [T, ld] fp32: y in columns 0 .. W - 1, x from column x0 on
// (both without biases); w_gates [parts, 2 B, B] in `dtype` (rows of r, then of i); out [T, W] in `dtype`.
DLGO_EXPORT int dlgo_rglru_step(const float* proj, int ld, int x0, const float* by, const float* bx, const float* w_taps,
                                const float* bc, const void* w_gates, const float* br, const float* bi, const float* lam,
                                const int* token_pos, const int* seq_slot, float* state, long long state_ld, void* out,
                                int dtype, int T, int W, int parts, int taps, float rate, cudaStream_t stream) {
  if (T <= 0) return DLGO_OK;
  const RglruShape s{W, parts, taps, rate};
  if (!rglru_ok(s)) return DLGO_ERR_SIZE;
#define ST_CALL(T_) launch_rglru_step<T_, T_>(proj, ld, x0, by, bx, w_taps, bc, (const T_*)w_gates, br, bi, lam, token_pos, seq_slot, \
                                              state, state_ld, (T_*)out, T, s, stream)
  if (dtype == DLGO_F32) return ST_CALL(float);
  if (dtype == DLGO_BF16) return ST_CALL(__nv_bfloat16);
#undef ST_CALL
  return DLGO_ERR_DTYPE;
}
