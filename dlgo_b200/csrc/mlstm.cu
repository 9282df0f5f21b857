// Matrix memory with exponential gates (mLSTM): per head, with log gates i_t and f_t and m_0 = 0,
//
//   m_t = max(f_t + m_(t-1), i_t)
//   S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T         S [N, P], fp32, zero at the start
//   n_t = exp(f_t + m_(t-1) - m_t) n_(t-1) + exp(i_t - m_t) k_t               n [N]
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
//
// where q carries a constant factor c (qk_scale), i = cap tanh((zi + bi) / cap) and f = logsigmoid(cap tanh((zf + bf) /
// cap)).  Once m is known this is the recurrence S <- f' S + d k v^T of ssd.cu / ssd_tc.cu with f' = exp(f + m_(t-1) -
// m_t) and d = exp(i - m_t), and the same on v = 1 for n.  A sequence's state row is [H N P of S | H N of n | H of m].
//
// mlstm_gates      prompts: the gates, the running maximum over each sequence, (d, f' or its logarithm) and m per token.
//                  m is a prefix of the maps m -> max(m + f, i), which compose to maps of the same form, so a block
//                  scans a sequence's tokens of one head in parallel.
// mlstm_norm_scan  prompts whose recurrence runs token by token: n_t . q_t, a warp per (sequence, head)
// mlstm_step       decoding: gates, S, n, read-out of one token per sequence in one launch
// mlstm_gate_norm  o from the read-out and n . q, divided by its root mean square per head, times a weight, a sigmoid gate
//                  and a constant; a decoding step's m moves into the state rows here (every reader of the old one ran
//                  in an earlier launch)
// Everything is fp32 in every precision.
#include "ssd_state.cuh"

#include <math_constants.h>

namespace dlgo {

struct MlstmShape {
  int H, N, P;
  __host__ __device__ long long norm_off() const { return (long long)H * N * P; }
  __host__ __device__ long long max_off() const { return (long long)H * N * (P + 1); }
};

__device__ __forceinline__ float ml_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float ml_capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float ml_log_forget(float z, float cap) { return -ml_softplus(-ml_capped(z, cap)); }

// ------------------------------------------------------------------------------- gates (prompts)
constexpr int MG_PER = 8;      // neighbouring tokens of a thread

__global__ void __launch_bounds__(256)
mlstm_gates_kernel(const float* zi, const float* zf, int ld, const float* __restrict__ bi, const float* __restrict__ bf,
                   float cap, const int* __restrict__ seqs, const int* __restrict__ seq_slot, float* state,
                   long long state_ld, float* steps, float* m_out, int log_decay, MlstmShape s) {
  pdl_launch_dependents();
  __shared__ float w_sum[8], w_max[8], carry;
  const int h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t0 = seqs[blockIdx.x * 3 + 1], count = seqs[blockIdx.x * 3 + 2];
  float* kept = state + (size_t)seq_slot[seqs[blockIdx.x * 3]] * state_ld + s.max_off() + h;
  const float b_i = bi[h], b_f = bf[h];
  pdl_wait();
  float m0 = *kept;
  for (int base = 0; base < count; base += blockDim.x * MG_PER) {
    const int b = base + threadIdx.x * MG_PER;
    float li[MG_PER], lf[MG_PER];
#pragma unroll
    for (int q = 0; q < MG_PER; ++q) {
      li[q] = -CUDART_INF_F;                        // (beyond the end: the map that changes nothing)
      lf[q] = 0.f;
      if (b + q < count) {
        li[q] = zi[(size_t)(t0 + b + q) * ld + h];
        lf[q] = zf[(size_t)(t0 + b + q) * ld + h];
      }
    }
    float sum = 0.f, top = -CUDART_INF_F;           // the thread's tokens as one map m -> max(m + sum, top)
#pragma unroll
    for (int q = 0; q < MG_PER; ++q) {
      if (b + q < count) {
        li[q] = ml_capped(li[q] + b_i, cap);
        lf[q] = ml_log_forget(lf[q] + b_f, cap);
        sum += lf[q];
        top = fmaxf(top + lf[q], li[q]);
      }
    }
    float isum = sum, itop = top;                   // inclusive over the warp's lanes
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float us = __shfl_up_sync(0xffffffffu, isum, o), ut = __shfl_up_sync(0xffffffffu, itop, o);
      if (lane >= o) {
        itop = fmaxf(ut + isum, itop);
        isum += us;
      }
    }
    if (lane == 31) {
      w_sum[warp] = isum;
      w_max[warp] = itop;
    }
    float psum = __shfl_up_sync(0xffffffffu, isum, 1), ptop = __shfl_up_sync(0xffffffffu, itop, 1);
    if (lane == 0) {
      psum = 0.f;
      ptop = -CUDART_INF_F;
    }
    __syncthreads();
    float m = m0;
    for (int w = 0; w < warp; ++w) m = fmaxf(m + w_sum[w], w_max[w]);
    m = fmaxf(m + psum, ptop);
#pragma unroll
    for (int q = 0; q < MG_PER; ++q) {
      if (b + q < count) {
        const float now = fmaxf(lf[q] + m, li[q]), decay = lf[q] + m - now;
        const size_t at = (size_t)(t0 + b + q) * s.H + h;
        *reinterpret_cast<float2*>(steps + at * 2) = make_float2(expf(li[q] - now), log_decay ? decay : expf(decay));
        m_out[at] = now;
        m = now;
      }
    }
    // the newest token's m, as it is (the state's scale), from the thread that holds that token
    const int end = min(count - base, (int)blockDim.x * MG_PER) - 1;
    if ((int)threadIdx.x == end / MG_PER) carry = m;
    __syncthreads();
    m0 = carry;
  }
  if (threadIdx.x == 0) *kept = m0;                 // (nobody else of this launch reads it)
}

// ------------------------------------------------------------------------------- n . q, token by token
constexpr int NS_WARPS = 4;

template <int NR>
__global__ void __launch_bounds__(NS_WARPS * 32)
mlstm_norm_scan_kernel(const float* k, const float* q, int ld, const float* steps, const int* __restrict__ seqs, int n_seqs,
                       const int* __restrict__ seq_slot, float* state, long long state_ld, float* nq, MlstmShape s) {
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, item = blockIdx.x * NS_WARPS + (threadIdx.x >> 5);
  if (item >= n_seqs * s.H) return;
  const int sq = item / s.H, h = item - sq * s.H;
  const int t0 = seqs[sq * 3 + 1], count = seqs[sq * 3 + 2];
  float* st = state + (size_t)seq_slot[seqs[sq * 3]] * state_ld + s.norm_off() + (size_t)h * s.N;
  pdl_wait();
  float n[NR], kn[NR], qn[NR];
  auto fetch = [&](int t, float2& step) {
    const size_t row = (size_t)t * ld + (size_t)h * s.N;
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int i = j * 32 + lane;
      kn[j] = i < s.N ? k[row + i] : 0.f;
      qn[j] = i < s.N ? q[row + i] : 0.f;
    }
    step = *reinterpret_cast<const float2*>(steps + ((size_t)t * s.H + h) * 2);
  };
#pragma unroll
  for (int j = 0; j < NR; ++j) n[j] = j * 32 + lane < s.N ? st[j * 32 + lane] : 0.f;
  float2 step;
  fetch(t0, step);
  for (int t = t0; t < t0 + count; ++t) {
    float dot = 0.f;
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      n[j] = fmaf(step.y, n[j], step.x * kn[j]);
      dot = fmaf(n[j], qn[j], dot);
    }
    if (t + 1 < t0 + count) fetch(t + 1, step);     // on its way while the lanes meet
    dot = warp_sum(dot);
    if (lane == 0) nq[(size_t)t * s.H + h] = dot;
  }
#pragma unroll
  for (int j = 0; j < NR; ++j)
    if (j * 32 + lane < s.N) st[j * 32 + lane] = n[j];
}

// ------------------------------------------------------------------------------- one token per sequence
// Blocks z < gridDim.z - 1: columns of S; the last: n and m.  proj row: v | k | q at columns 0, H P, H (P + N); log-gate
// logits at zi / zf.
template <int RS>
__global__ void __launch_bounds__(RS <= 8 ? 128 : 16 * RS, RS <= 8 ? 4 : (RS == 16 ? 2 : 1))
mlstm_step_kernel(const float* proj, const float* zi, const float* zf, int ld, const float* __restrict__ bi,
                  const float* __restrict__ bf, float cap, const int* __restrict__ seq_slot, float* state,
                  long long state_ld, float* out, int ldo, float* nq, float* m_out, MlstmShape s, int vec) {
  using TL = SsdTile<RS>;
  constexpr int NPAD = TL::NPAD;
  pdl_launch_dependents();
  __shared__ __align__(16) float row[2 * NPAD + TL::COLS];         // k | q | v
  __shared__ float red[32];
  const int t = blockIdx.x, h = blockIdx.y, N = s.N, P = s.P;
  float* srow = state + (size_t)seq_slot[t] * state_ld;
  const float* pr = proj + (size_t)t * ld;
  const float* kp = pr + (size_t)s.H * P + (size_t)h * N;
  const float* qp = kp + (size_t)s.H * N;
  const float b_i = bi[h], b_f = bf[h];
  const bool normalizer = blockIdx.z == gridDim.z - 1;
  const int r = threadIdx.x % RS, cl = (threadIdx.x / RS) * 4;
  const int e0 = blockIdx.z * TL::COLS, e = e0 + cl, nx = normalizer ? 0 : min(TL::COLS, P - e0);
  float* st = srow + (size_t)h * N * P;
  for (int i = threadIdx.x; i < 2 * NPAD + TL::COLS; i += blockDim.x) row[i] = 0.f;
  __syncthreads();
  pdl_wait();
  f32x2 S[8][4];
  if (!normalizer) {
    ssd_load_state<RS>(S, st, N, P, e, r, vec);                    // in flight while the rows arrive
    for (int i = threadIdx.x; i < 2 * N + nx; i += blockDim.x) {
      if (i < N) row[i] = kp[i];
      else if (i < 2 * N) row[NPAD + i - N] = qp[i - N];
      else row[2 * NPAD + i - 2 * N] = pr[h * P + e0 + i - 2 * N];
    }
  }
  const float li = ml_capped(zi[(size_t)t * ld + h] + b_i, cap), lf = ml_log_forget(zf[(size_t)t * ld + h] + b_f, cap);
  const float m = srow[s.max_off() + h], now = fmaxf(lf + m, li);
  const float f = expf(lf + m - now), d = expf(li - now);
  if (normalizer) {
    float* n = srow + s.norm_off() + (size_t)h * N;
    float dot = 0.f;
    for (int i = threadIdx.x; i < N; i += blockDim.x) {
      const float v = fmaf(f, n[i], d * kp[i]);
      n[i] = v;
      dot = fmaf(v, qp[i], dot);
    }
    dot = block_sum(dot, red);
    if (threadIdx.x == 0) {
      nq[(size_t)t * s.H + h] = dot;
      m_out[(size_t)t * s.H + h] = now;             // (into the state row by the launch behind: others still read the old one)
    }
    return;
  }
  __syncthreads();
  float4 v = *reinterpret_cast<const float4*>(row + 2 * NPAD + cl);
  v.x *= d; v.y *= d; v.z *= d; v.w *= d;
  float y[4] = {0.f, 0.f, 0.f, 0.f};
  ssd_token<RS, true>(S, row, row + NPAD, f, v, r, y);
  ssd_store_state<RS>(S, st, N, P, e, r, vec);
  ssd_meet<RS>(y, r);
  ssd_write<RS>(y, row + 2 * NPAD + cl, 0.f, out + (size_t)t * ldo + (size_t)h * P, e, P, r);
}

// ------------------------------------------------------------------------------- read-out, norm and gate
constexpr int MN_WARPS = 4;

__device__ __forceinline__ void mn_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void mn_store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 h[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(h);
}
__device__ __forceinline__ float ml_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// A warp per (token, head).  NV > 0: heads of up to 128 NV numbers, a multiple of four, held in registers; NV 0: any.
template <typename TO, int NV>
__global__ void __launch_bounds__(MN_WARPS * 32)
mlstm_gate_norm_kernel(const float* o, int ldo, const float* nq, const float* m_now, float qk_scale, const float* g, int ldg,
                       const float* __restrict__ w, float eps, float out_scale, TO* out, int T,
                       const int* __restrict__ seq_slot, float* state, long long state_ld, int store_m, MlstmShape s) {
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, P = s.P;
  const long long item = (long long)blockIdx.x * MN_WARPS + (threadIdx.x >> 5);
  if (item >= (long long)T * s.H) return;
  const int t = (int)(item / s.H), h = (int)(item - (long long)t * s.H);
  const float* wp = w + (size_t)h * P;
  constexpr int R = NV > 0 ? NV : 1;
  float4 u[R], z[R], wv[R];
  if (NV > 0) {
#pragma unroll
    for (int v = 0; v < R; ++v) {
      const int i = (v * 32 + lane) * 4;
      if (i < P) wv[v] = *reinterpret_cast<const float4*>(wp + i);
    }
  }
  pdl_wait();
  const float* orow = o + (size_t)t * ldo + (size_t)h * P;
  const float* grow = g + (size_t)t * ldg + (size_t)h * P;
  TO* dst = out + ((size_t)t * s.H + h) * P;
  const float m = m_now[item];
  const float c = qk_scale / (fmaxf(fabsf(nq[item] * qk_scale), expf(-m)) + 1e-6f);
  float ss = 0.f;
  if (NV > 0) {
#pragma unroll
    for (int v = 0; v < R; ++v) {
      const int i = (v * 32 + lane) * 4;
      if (i < P) {
        u[v] = *reinterpret_cast<const float4*>(orow + i);
        z[v] = *reinterpret_cast<const float4*>(grow + i);
        u[v].x *= c; u[v].y *= c; u[v].z *= c; u[v].w *= c;
        ss += (u[v].x * u[v].x + u[v].y * u[v].y) + (u[v].z * u[v].z + u[v].w * u[v].w);
      }
    }
  } else {
    for (int i = lane; i < P; i += 32) ss = fmaf(orow[i] * c, orow[i] * c, ss);
  }
  const float sc = out_scale / sqrtf(warp_sum(ss) / (float)P + eps);
  if (NV > 0) {
#pragma unroll
    for (int v = 0; v < R; ++v) {
      const int i = (v * 32 + lane) * 4;
      if (i < P)
        mn_store4(dst + i, make_float4(u[v].x * sc * wv[v].x * ml_sigmoid(z[v].x), u[v].y * sc * wv[v].y * ml_sigmoid(z[v].y),
                                       u[v].z * sc * wv[v].z * ml_sigmoid(z[v].z), u[v].w * sc * wv[v].w * ml_sigmoid(z[v].w)));
    }
  } else {
    for (int i = lane; i < P; i += 32) dst[i] = from_float<TO>(orow[i] * c * sc * wp[i] * ml_sigmoid(grow[i]));
  }
  if (store_m && lane == 0) state[(size_t)seq_slot[t] * state_ld + s.max_off() + h] = m;
}

static bool mlstm_ok(const MlstmShape& s) { return s.H > 0 && s.H <= 65535 && s.N > 0 && s.N <= 512 && s.P > 0; }

template <typename TO>
static int launch_mlstm_gate_norm(const float* o, int ldo, const float* nq, const float* m_now, float qk_scale, const float* g,
                                  int ldg, const float* w, float eps, float out_scale, TO* out, int T, const int* seq_slot,
                                  float* state, long long state_ld, int store_m, const MlstmShape& s, cudaStream_t stream) {
  const long long blocks = ((long long)T * s.H + MN_WARPS - 1) / MN_WARPS;
  if (blocks > 0x7fffffffLL) return DLGO_ERR_SIZE;
  const bool four = ((s.P | ldo | ldg) & 3) == 0 && (((uintptr_t)o | (uintptr_t)g | (uintptr_t)w | (uintptr_t)out) & 15) == 0;
#define MN_ARGS dim3((unsigned)blocks), dim3(MN_WARPS * 32), 0, stream, o, ldo, nq, m_now, qk_scale, g, ldg, w, eps, out_scale, \
                out, T, seq_slot, state, state_ld, store_m, s
  if (four && s.P <= 128) launch_kernel(mlstm_gate_norm_kernel<TO, 1>, MN_ARGS);
  else if (four && s.P <= 256) launch_kernel(mlstm_gate_norm_kernel<TO, 2>, MN_ARGS);
  else if (four && s.P <= 512) launch_kernel(mlstm_gate_norm_kernel<TO, 4>, MN_ARGS);
  else launch_kernel(mlstm_gate_norm_kernel<TO, 0>, MN_ARGS);
#undef MN_ARGS
  return launch_status();
}

}  // namespace dlgo

using namespace dlgo;

// zi, zf [T, ld] fp32 (H columns each: the log gates' logits), bi, bf [H]; seqs [n_seqs, 3] (sequence, first packed token,
// count): every sequence of the step, `longest` its largest count; steps [T, H, 2]: d and f' (log_decay: its logarithm);
// m_out [T, H]; m in the state rows is read and replaced.
DLGO_EXPORT int dlgo_mlstm_gates(const float* zi, const float* zf, int ld, const float* bi, const float* bf, float cap,
                                 const int* seqs, int n_seqs, int longest, const int* seq_slot, float* state,
                                 long long state_ld, float* steps, float* m_out, int log_decay, int H, int N, int P,
                                 cudaStream_t stream) {
  if (n_seqs <= 0) return DLGO_OK;
  const MlstmShape s{H, N, P};
  if (!mlstm_ok(s) || !(cap > 0.f)) return DLGO_ERR_SIZE;
  const int threads = longest <= 32 * MG_PER ? 32 : (longest <= 128 * MG_PER ? 128 : 256);
  launch_kernel(mlstm_gates_kernel, dim3(n_seqs, H), dim3(threads), 0, stream, zi, zf, ld, bi, bf, cap, seqs, seq_slot, state,
                state_ld, steps, m_out, log_decay, s);
  return launch_status();
}

// k, q [T, ld] fp32 (H heads of N), steps of dlgo_mlstm_gates with f' itself; nq [T, H] = n_t . q_t
DLGO_EXPORT int dlgo_mlstm_norm_scan(const float* k, const float* q, int ld, const float* steps, const int* seqs, int n_seqs,
                                     const int* seq_slot, float* state, long long state_ld, float* nq, int H, int N, int P,
                                     cudaStream_t stream) {
  if (n_seqs <= 0) return DLGO_OK;
  const MlstmShape s{H, N, P};
  if (!mlstm_ok(s)) return DLGO_ERR_SIZE;
  const dim3 grid((n_seqs * H + NS_WARPS - 1) / NS_WARPS), block(NS_WARPS * 32);
#define NS_ARGS grid, block, 0, stream, k, q, ld, steps, seqs, n_seqs, seq_slot, state, state_ld, nq, s
  if (N <= 32) launch_kernel(mlstm_norm_scan_kernel<1>, NS_ARGS);
  else if (N <= 64) launch_kernel(mlstm_norm_scan_kernel<2>, NS_ARGS);
  else if (N <= 128) launch_kernel(mlstm_norm_scan_kernel<4>, NS_ARGS);
  else if (N <= 256) launch_kernel(mlstm_norm_scan_kernel<8>, NS_ARGS);
  else launch_kernel(mlstm_norm_scan_kernel<16>, NS_ARGS);
#undef NS_ARGS
  return launch_status();
}

// One token per sequence (token t belongs to sequence t).  proj [T, ld] fp32: v (H P) | k (H N) | q (H N) | ...; zi, zf
// with the same row stride; out [T, ldo >= H P] = S^T q, nq [T, H] = n . q, m_out [T, H]; S and n move on in the state
// rows, m is left to dlgo_mlstm_gate_norm.
DLGO_EXPORT int dlgo_mlstm_step(const float* proj, const float* zi, const float* zf, int ld, const float* bi, const float* bf,
                                float cap, const int* seq_slot, float* state, long long state_ld, float* out, int ldo,
                                float* nq, float* m_out, int T, int H, int N, int P, cudaStream_t stream) {
  if (T <= 0) return DLGO_OK;
  const MlstmShape s{H, N, P};
  if (!mlstm_ok(s) || !(cap > 0.f)) return DLGO_ERR_SIZE;
  const int vec = (P & 3) == 0 && (state_ld & 3) == 0 && ((uintptr_t)state & 15) == 0;
#define STEP_LAUNCH(RS) \
  launch_kernel(mlstm_step_kernel<RS>, dim3(T, H, ssd_col_blocks<RS>(P) + 1), ssd_block<RS>(P), 0, stream, proj, zi, zf, ld, bi, \
                bf, cap, seq_slot, state, state_ld, out, ldo, nq, m_out, s, vec)
  switch (ssd_row_split(N)) {
    case 1: STEP_LAUNCH(1); break;
    case 2: STEP_LAUNCH(2); break;
    case 4: STEP_LAUNCH(4); break;
    case 8: STEP_LAUNCH(8); break;
    case 16: STEP_LAUNCH(16); break;
    default: STEP_LAUNCH(32); break;
  }
#undef STEP_LAUNCH
  return launch_status();
}

// o [T, ldo >= H P] = S^T q, nq and m_now [T, H], g [T, ldg >= H P] (gate logits), w [H P], all fp32; out [T, H P] in
// `dtype`.  `store_m` (one token per sequence): m_now goes into the state rows.
DLGO_EXPORT int dlgo_mlstm_gate_norm(const float* o, int ldo, const float* nq, const float* m_now, float qk_scale,
                                     const float* g, int ldg, const float* w, float eps, float out_scale, void* out, int dtype,
                                     int T, const int* seq_slot, float* state, long long state_ld, int store_m, int H, int N,
                                     int P, cudaStream_t stream) {
  if (T <= 0) return DLGO_OK;
  const MlstmShape s{H, N, P};
  if (!mlstm_ok(s)) return DLGO_ERR_SIZE;
#define MN_ARGS(T_) o, ldo, nq, m_now, qk_scale, g, ldg, w, eps, out_scale, (T_*)out, T, seq_slot, state, state_ld, store_m, s, stream
  if (dtype == DLGO_F32) return launch_mlstm_gate_norm<float>(MN_ARGS(float));
  if (dtype == DLGO_BF16) return launch_mlstm_gate_norm<__nv_bfloat16>(MN_ARGS(__nv_bfloat16));
#undef MN_ARGS
  return DLGO_ERR_DTYPE;
}
