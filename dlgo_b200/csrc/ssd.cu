// State-space mixing with a scalar decay per head and token (the recurrence of Mamba-2), its short convolution and its
// gated group norm.
//
// One projection row per token holds [z: H P | x: H P | B: G N | C: G N | dt: H] (fp32).  With a the silu:
//   conv:   (x | B | C)_t <- a(bias + sum_j taps[:, j] u_(t - n + 1 + j))   per channel, u = 0 before a sequence's start
//   step:   d_t = softplus(dt_t + dt_bias),  f_t = exp(-exp(A_log) d_t)     per head
//   state:  S_t = f_t S_(t-1) + d_t B_t x_t^T                               S [N, P] per head, fp32, zero at the start
//   out:    y_t = S_t^T C_t + D x_t                                         head h reads B and C of group h / (H / G)
//   norm:   u = y * a(z);  each of `groups` equal parts of u divided by its root mean square, then times w
// A sequence's state row is [H N P numbers of S | (n - 1) inputs of the convolution, oldest first], fp32, `state_ld`
// floats apart, and is carried from step to step.
//
// ssd_conv       prompts: convolution and silu of every channel, d and f of every head, for all tokens of the step
// ssd_segments   prompts: a sequence's tokens are cut into segments that run side by side
//                  LOCAL   every segment but a sequence's last runs from a zero state: its end state L_j, and the
//                          product F_j of its decays
//                  carry   starts[j] = F_(j-1) starts[j-1] + L_(j-1) from the stored state, element by element
//                  FULL    every segment walks its tokens from its start; the last one stores the sequence's new state
//                with one segment per sequence FULL runs alone from the stored state
// ssd_step       decoding: convolution, step, state and output of one token per sequence in one launch
// ssd_gate_norm  gate and norm; blocks of the same launch move the convolution's inputs into the state rows (every
//                reader of the old ones ran in an earlier launch)
//
// The state kernels share one layout (ssd_state.cuh).  Everything is fp32 in every precision.
#include "ssd.cuh"
#include "ssd_state.cuh"
#include "async_copy.cuh"

namespace dlgo {

__device__ __forceinline__ float ssd_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float ssd_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// The input of channel c at packed token `tok` of sequence `seq` (tok may lie before the sequence's first token of
// this step; `first` is that token): a projected number, or one kept from an earlier step.
__device__ __forceinline__ float conv_input(const float* xbc, int ld, int tok, int first, int c, const float* kept,
                                            int taps, int channels) {
  if (tok >= first) return xbc[(size_t)tok * ld + c];
  return kept[(size_t)(taps - 1 + tok - first) * channels + c];
}

// ------------------------------------------------------------------------------- convolution (prompts)
constexpr int SC_THREADS = 128;

__device__ __forceinline__ void conv_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void conv_store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 h[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(h);
}

// A thread owns W neighbouring channels and walks its tile's tokens with the taps' reach in registers (TAPS > 0) or
// reads every tap from memory (TAPS 0: any number of taps).
template <typename TO, int TAPS, int W>
__global__ void __launch_bounds__(SC_THREADS)
ssd_conv_kernel(const float* proj, int ld, const float* __restrict__ w_taps, const float* __restrict__ w_bias,
                const float* __restrict__ dt_bias, const float* __restrict__ a_log, const int* __restrict__ tiles,
                const int* __restrict__ token_seq, const int* __restrict__ seq_slot, const float* state,
                long long state_ld, TO* out, int ldo, float* steps, int log_decay, SsdShape s) {
  pdl_launch_dependents();
  const int tile = blockIdx.x;
  const int seq = tiles[tile * 3 + 0], t0 = tiles[tile * 3 + 1], count = tiles[tile * 3 + 2];
  const int C = s.channels(), n_taps = TAPS > 0 ? TAPS : s.taps;
  if (blockIdx.y == gridDim.y - 1) {               // the heads' steps and decays
    pdl_wait();
    const float* dt = proj + s.inner() + C;
    for (int i = threadIdx.x; i < count * s.H; i += SC_THREADS) {
      const int t = t0 + i / s.H, h = i % s.H;
      const float d = ssd_softplus(dt[(size_t)t * ld + h] + dt_bias[h]);
      steps[((size_t)t * s.H + h) * 2] = d;
      const float lf = -expf(a_log[h]) * d;
      steps[((size_t)t * s.H + h) * 2 + 1] = log_decay ? lf : expf(lf);
    }
    return;
  }
  const int c = (blockIdx.y * SC_THREADS + threadIdx.x) * W;
  if (c >= C) return;
  int first = t0;                                  // the sequence's first token of this step, if within the taps' reach
  while (first > 0 && first > t0 - n_taps + 1 && token_seq[first - 1] == seq) --first;
  const float* kept = state + (size_t)seq_slot[seq] * state_ld + s.conv_off();
  const float* xbc = proj + s.inner();
  float bias[W];
#pragma unroll
  for (int k = 0; k < W; ++k) bias[k] = w_bias[c + k];
  if (TAPS > 0) {
    constexpr int R = TAPS > 0 ? TAPS : 1, FLY = 8;
    float tap[R][W], u[R][W];
#pragma unroll
    for (int k = 0; k < W; ++k) {
      if (R == 4 && W == 4) {                      // (four taps of a channel: 16 bytes)
        const float4 v = *reinterpret_cast<const float4*>(w_taps + (size_t)(c + k) * 4);
        tap[0][k] = v.x; tap[1 % R][k] = v.y; tap[2 % R][k] = v.z; tap[3 % R][k] = v.w;
      } else {
#pragma unroll
        for (int j = 0; j < R; ++j) tap[j][k] = w_taps[(size_t)(c + k) * R + j];
      }
    }
    pdl_wait();
#pragma unroll
    for (int j = 0; j < R - 1; ++j) {
#pragma unroll
      for (int k = 0; k < W; ++k) u[j][k] = conv_input(xbc, ld, t0 - R + 1 + j, first, c + k, kept, R, C);
    }
    for (int tb = 0; tb < count; tb += FLY) {
      float in[FLY][W];                            // several tokens' fetches in flight
#pragma unroll
      for (int q = 0; q < FLY; ++q) {
        const float* src = xbc + (size_t)(t0 + min(tb + q, count - 1)) * ld + c;
        if (W == 4) {
          const float4 v = *reinterpret_cast<const float4*>(src);
          in[q][0] = v.x; in[q][1 % W] = v.y; in[q][2 % W] = v.z; in[q][3 % W] = v.w;
        } else {
          in[q][0] = src[0];
        }
      }
#pragma unroll
      for (int q = 0; q < FLY; ++q) {
        if (tb + q >= count) break;
        float y[W];
#pragma unroll
        for (int k = 0; k < W; ++k) {
          u[R - 1][k] = in[q][k];
          float a = bias[k];
#pragma unroll
          for (int j = 0; j < R; ++j) a = fmaf(tap[j][k], u[j][k], a);
          y[k] = ssd_silu(a);
#pragma unroll
          for (int j = 0; j < R - 1; ++j) u[j][k] = u[j + 1][k];
        }
        TO* dst = out + (size_t)(t0 + tb + q) * ldo + c;
        if (W == 4) conv_store4(dst, make_float4(y[0], y[1 % W], y[2 % W], y[3 % W]));
        else dst[0] = from_float<TO>(y[0]);
      }
    }
    return;
  }
  pdl_wait();
  for (int t = t0; t < t0 + count; ++t) {
#pragma unroll
    for (int k = 0; k < W; ++k) {
      float a = bias[k];
      for (int j = 0; j < n_taps; ++j)
        a = fmaf(w_taps[(size_t)(c + k) * n_taps + j], conv_input(xbc, ld, t - n_taps + 1 + j, first, c + k, kept, n_taps, C), a);
      out[(size_t)t * ldo + c + k] = from_float<TO>(ssd_silu(a));
    }
  }
}

enum { SSD_LOCAL = 0, SSD_FULL = 1 };


// tokens arrive in chunks through a ring of two shared-memory buffers, one chunk ahead of the products
template <int RS, int MODE>
__global__ void __launch_bounds__(RS <= 8 ? 128 : 16 * RS)
ssd_segments_kernel(const float* xbc, int ld, const float* steps, const float* __restrict__ D,
                    const int* __restrict__ tiles, int n_tiles, const int* __restrict__ seq_slot, float* state,
                    long long state_ld, float* seg, float* seg_decay, float* out, int ldo, SsdShape s, int direct,
                    int vec) {
  using TL = SsdTile<RS>;
  constexpr int CH = TL::CH, ROW = TL::ROW, NPAD = TL::NPAD;
  pdl_launch_dependents();
  extern __shared__ __align__(16) float ring[];                    // [2][CH][ROW]
  const int tile = blockIdx.x, h = blockIdx.y;
  const int seq = tiles[tile * 3 + 0], t0 = tiles[tile * 3 + 1], count = tiles[tile * 3 + 2];
  const bool last = tile + 1 == n_tiles || tiles[(tile + 1) * 3] != seq;
  if (MODE == SSD_LOCAL && last) return;                           // nobody starts from its end
  const int N = s.N, P = s.P, g = h / (s.H / s.G);
  const int r = threadIdx.x % RS, cl = (threadIdx.x / RS) * 4;     // this thread's row group and first column of the block
  const int e0 = blockIdx.z * TL::COLS, e = e0 + cl;
  const int nx = min(TL::COLS, P - e0);
  float* st = state + (size_t)seq_slot[seq] * state_ld + (size_t)h * N * P;
  float* sg = seg == nullptr ? nullptr : seg + ((size_t)tile * s.H + h) * N * P;
  const float Dh = D != nullptr ? D[h] : 0.f;
  for (int i = threadIdx.x; i < 2 * CH * ROW; i += blockDim.x) ring[i] = 0.f;      // (rows beyond N stay zero)
  __syncthreads();
  pdl_wait();
  const int b_off = s.inner() + g * N, c_off = b_off + s.G * N, x_off = h * P + e0;
  auto load_chunk = [&](int c, float* buf) {
    const int tok0 = t0 + c * CH, nt = min(CH, count - c * CH);
    const int unit = vec ? 4 : 1, nb = N / unit, per = 2 * nb + (nx + unit - 1) / unit;
    for (int i = threadIdx.x; i < nt * per; i += blockDim.x) {
      const int t = i / per, p = i - t * per;
      const float* row = xbc + (size_t)(tok0 + t) * ld;
      float* dst = buf + t * ROW;
      const float* src;
      if (p < nb) { src = row + b_off + p * unit; dst += p * unit; }
      else if (p < 2 * nb) { src = row + c_off + (p - nb) * unit; dst += NPAD + (p - nb) * unit; }
      else { src = row + x_off + (p - 2 * nb) * unit; dst += 2 * NPAD + (p - 2 * nb) * unit; }
      if (vec) copy16_async(dst, src);
      else copy4_async(dst, src);
    }
    for (int i = threadIdx.x; i < nt * 2; i += blockDim.x)
      copy4_async(buf + (i >> 1) * ROW + 2 * NPAD + TL::COLS + (i & 1), steps + ((size_t)(tok0 + (i >> 1)) * s.H + h) * 2 + (i & 1));
    copies_commit();
  };
  const int n_chunks = (count + CH - 1) / CH;
  load_chunk(0, ring);
  f32x2 S[8][4];
  if (MODE == SSD_LOCAL) {
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int k = 0; k < 4; ++k) S[j][k] = 0ull;
  } else {
    ssd_load_state<RS>(S, direct ? st : sg, N, P, e, r, vec);
  }
  float prod = 1.f;
  for (int c = 0; c < n_chunks; ++c) {
    float* buf = ring + (c & 1) * CH * ROW;
    if (c + 1 < n_chunks) {
      load_chunk(c + 1, ring + ((c + 1) & 1) * CH * ROW);          // (its last readers passed the barrier that ended chunk c - 1)
      copies_wait<1>();
    } else {
      copies_wait<0>();
    }
    __syncthreads();
    const int nt = min(CH, count - c * CH);
    for (int t = 0; t < nt; ++t) {
      const float* cur = buf + t * ROW;
      const float d = cur[2 * NPAD + TL::COLS], f = cur[2 * NPAD + TL::COLS + 1];
      float4 v = *reinterpret_cast<const float4*>(cur + 2 * NPAD + cl);
      v.x *= d; v.y *= d; v.z *= d; v.w *= d;
      float y[4] = {0.f, 0.f, 0.f, 0.f};
      ssd_token<RS, MODE == SSD_FULL>(S, cur, cur + NPAD, f, v, r, y);
      if (MODE == SSD_LOCAL) {
        prod *= f;
      } else {
        ssd_meet<RS>(y, r);
        ssd_write<RS>(y, cur + 2 * NPAD + cl, Dh, out + (size_t)(t0 + c * CH + t) * ldo + (size_t)h * P, e, P, r);
      }
    }
    __syncthreads();                                               // the buffer is free for the chunk after next
  }
  if (MODE == SSD_LOCAL) {
    ssd_store_state<RS>(S, sg, N, P, e, r, vec);
    if (threadIdx.x == 0 && blockIdx.z == 0) seg_decay[(size_t)tile * s.H + h] = prod;
  } else if (last) {
    ssd_store_state<RS>(S, st, N, P, e, r, vec);
  }
}

// ------------------------------------------------------------------------------- one token per sequence
template <int RS>
__global__ void __launch_bounds__(RS <= 8 ? 128 : 16 * RS, RS <= 8 ? 4 : (RS == 16 ? 2 : 1))
ssd_step_kernel(const float* proj, int ld, const float* __restrict__ w_taps, const float* __restrict__ w_bias,
                const float* __restrict__ dt_bias, const float* __restrict__ a_log, const float* __restrict__ D,
                const int* __restrict__ seq_slot, float* state, long long state_ld, float* out, int ldo, SsdShape s,
                int vec) {
  using TL = SsdTile<RS>;
  constexpr int NPAD = TL::NPAD;
  pdl_launch_dependents();
  __shared__ __align__(16) float row[2 * NPAD + TL::COLS];         // B | C | x
  const int t = blockIdx.x, h = blockIdx.y;
  const int N = s.N, P = s.P, g = h / (s.H / s.G), C = s.channels();
  const int r = threadIdx.x % RS, cl = (threadIdx.x / RS) * 4;
  const int e0 = blockIdx.z * TL::COLS, e = e0 + cl;
  const int nx = min(TL::COLS, P - e0);
  float* srow = state + (size_t)seq_slot[t] * state_ld;
  float* st = srow + (size_t)h * N * P;
  const float* kept = srow + s.conv_off();
  const float Dh = D[h], rate = expf(a_log[h]), db = dt_bias[h];
  for (int i = threadIdx.x; i < 2 * NPAD + TL::COLS; i += blockDim.x) row[i] = 0.f;
  __syncthreads();
  pdl_wait();
  f32x2 S[8][4];
  ssd_load_state<RS>(S, st, N, P, e, r, vec);                      // in flight while the convolution is formed
  const float* pr = proj + (size_t)t * ld + s.inner();
  const int b_off = s.inner() + g * N, c_off = b_off + s.G * N, x_off = h * P + e0;
  for (int i = threadIdx.x; i < 2 * N + nx; i += blockDim.x) {
    int c, dst;
    if (i < N) { c = b_off + i; dst = i; }
    else if (i < 2 * N) { c = c_off + i - N; dst = NPAD + i - N; }
    else { c = x_off + i - 2 * N; dst = 2 * NPAD + i - 2 * N; }
    const float now = pr[c];
    float a = w_bias[c];
    for (int j = 0; j < s.taps - 1; ++j) a = fmaf(w_taps[(size_t)c * s.taps + j], kept[(size_t)j * C + c], a);
    row[dst] = ssd_silu(fmaf(w_taps[(size_t)c * s.taps + s.taps - 1], now, a));
  }
  const float d = ssd_softplus(pr[C + h] + db), f = expf(-rate * d);
  __syncthreads();
  float4 v = *reinterpret_cast<const float4*>(row + 2 * NPAD + cl);
  v.x *= d; v.y *= d; v.z *= d; v.w *= d;
  float y[4] = {0.f, 0.f, 0.f, 0.f};
  ssd_token<RS, true>(S, row, row + NPAD, f, v, r, y);
  ssd_store_state<RS>(S, st, N, P, e, r, vec);
  ssd_meet<RS>(y, r);
  ssd_write<RS>(y, row + 2 * NPAD + cl, Dh, out + (size_t)t * ldo + (size_t)h * P, e, P, r);
}

// ------------------------------------------------------------------------------- gate and norm
// The convolution's inputs that a sequence's next tokens reach back to, moved into its state row: blocks behind those of
// the norm, a thread per (sequence, channel).  `seqs` [.., 3]: (sequence, first packed token, count) of the step.
constexpr int KEEP_REGS = 8;
__device__ __forceinline__ void keep_conv_inputs(const float* proj, int ld, const int* seqs, const int* seq_slot,
                                                 float* state, long long state_ld, const SsdShape& s, int block) {
  const int C = s.channels(), per_seq = (C + blockDim.x - 1) / blockDim.x, keep = s.taps - 1;
  const int q = block / per_seq, c = (block - q * per_seq) * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int seq = seqs[q * 3], end = seqs[q * 3 + 1] + seqs[q * 3 + 2];
  const int here = min(seqs[q * 3 + 2], keep);     // tokens of this step that the new row takes
  float* kept = state + (size_t)seq_slot[seq] * state_ld + s.conv_off() + c;
  const float* xbc = proj + s.inner() + c;
  // entry j is the input `keep - j` tokens before the sequence's next one; entries that stay move down by `here`
  for (int jb = 0; jb < keep; jb += KEEP_REGS) {   // (ascending: an old entry is read before it is overwritten)
    float v[KEEP_REGS];
#pragma unroll
    for (int u = 0; u < KEEP_REGS; ++u) {
      const int j = jb + u;
      if (j < keep) v[u] = j >= keep - here ? xbc[(size_t)(end - keep + j) * ld] : kept[(size_t)(j + here) * C];
    }
#pragma unroll
    for (int u = 0; u < KEEP_REGS; ++u)
      if (jb + u < keep) kept[(size_t)(jb + u) * C] = v[u];
  }
}

// A warp per (token, part) with the part's gated numbers in registers: parts of up to 128 NV numbers, a multiple of 4.
constexpr int GN_WARPS = 4;
template <typename TO, int NV>
__global__ void __launch_bounds__(GN_WARPS * 32)
ssd_gate_norm_warp_kernel(const float* y, int ldy, const float* proj, int ld, const float* __restrict__ w, TO* out, int groups,
                          float eps, const int* __restrict__ seqs, int T, int norm_blocks, const int* __restrict__ seq_slot,
                          float* state, long long state_ld, SsdShape s) {
  pdl_launch_dependents();
  if ((int)blockIdx.x >= norm_blocks) {
    pdl_wait();
    keep_conv_inputs(proj, ld, seqs, seq_slot, state, state_ld, s, blockIdx.x - norm_blocks);
    return;
  }
  const int lane = threadIdx.x & 31, n = s.inner() / groups;
  const long long item = (long long)blockIdx.x * GN_WARPS + (threadIdx.x >> 5);
  if (item >= (long long)T * groups) return;
  const int t = (int)(item / groups), part = (int)(item - (long long)t * groups);
  float4 wv[NV], u[NV], z[NV];
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = (v * 32 + lane) * 4;
    if (i < n) wv[v] = *reinterpret_cast<const float4*>(w + (size_t)part * n + i);
  }
  pdl_wait();
  const float* yr = y + (size_t)t * ldy + (size_t)part * n;
  const float* zr = proj + (size_t)t * ld + (size_t)part * n;
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = (v * 32 + lane) * 4;
    if (i < n) {
      u[v] = *reinterpret_cast<const float4*>(yr + i);
      z[v] = *reinterpret_cast<const float4*>(zr + i);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < NV; ++v)
    if ((v * 32 + lane) * 4 < n) {
      u[v].x *= ssd_silu(z[v].x); u[v].y *= ssd_silu(z[v].y); u[v].z *= ssd_silu(z[v].z); u[v].w *= ssd_silu(z[v].w);
      ss += (u[v].x * u[v].x + u[v].y * u[v].y) + (u[v].z * u[v].z + u[v].w * u[v].w);
    }
  const float sc = 1.0f / sqrtf(warp_sum(ss) / (float)n + eps);
  TO* dst = out + (size_t)t * s.inner() + (size_t)part * n;
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = (v * 32 + lane) * 4;
    if (i < n)
      conv_store4(dst + i, make_float4(u[v].x * sc * wv[v].x, u[v].y * sc * wv[v].y, u[v].z * sc * wv[v].z, u[v].w * sc * wv[v].w));
  }
}

// A block per (token, part), parts of any size.  `stash`: the part's gated numbers stay in shared memory between the passes.
template <typename TO>
__global__ void __launch_bounds__(512)
ssd_gate_norm_kernel(const float* y, int ldy, const float* proj, int ld, const float* __restrict__ w, TO* out, int groups,
                     float eps, const int* __restrict__ seqs, int norm_blocks, const int* __restrict__ seq_slot, float* state,
                     long long state_ld, SsdShape s, int stash) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float u_s[];
  __shared__ float red[32];
  pdl_wait();
  if ((int)blockIdx.x >= norm_blocks) {
    keep_conv_inputs(proj, ld, seqs, seq_slot, state, state_ld, s, blockIdx.x - norm_blocks);
    return;
  }
  const int t = blockIdx.x / groups, part = blockIdx.x - t * groups, n = s.inner() / groups;
  const float* yr = y + (size_t)t * ldy + (size_t)part * n;
  const float* zr = proj + (size_t)t * ld + (size_t)part * n;
  float ss = 0.f;
  const bool four = n % 4 == 0 && ldy % 4 == 0 && ld % 4 == 0 && ((uintptr_t)y & 15) == 0 && ((uintptr_t)proj & 15) == 0;
  if (stash && four) {
    for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
      const float4 a = *reinterpret_cast<const float4*>(yr + i), z = *reinterpret_cast<const float4*>(zr + i);
      const float4 u = make_float4(a.x * ssd_silu(z.x), a.y * ssd_silu(z.y), a.z * ssd_silu(z.z), a.w * ssd_silu(z.w));
      ss += (u.x * u.x + u.y * u.y) + (u.z * u.z + u.w * u.w);
      *reinterpret_cast<float4*>(u_s + i) = u;
    }
  } else {
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
      const float u = yr[i] * ssd_silu(zr[i]);
      ss = fmaf(u, u, ss);
      if (stash) u_s[i] = u;
    }
  }
  const float sc = 1.0f / sqrtf(block_sum(ss, red) / (float)n + eps);
  TO* dst = out + (size_t)t * s.inner() + (size_t)part * n;
  const float* wp = w + (size_t)part * n;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float u = stash ? u_s[i] : yr[i] * ssd_silu(zr[i]);      // (block_sum's barriers lie between u_s's writes and reads)
    dst[i] = from_float<TO>(u * sc * wp[i]);
  }
}

template <typename TO>
static int launch_ssd_gate_norm(const float* y, int ldy, const float* proj, int ld, const float* w, TO* out, int groups,
                                float eps, const int* seqs, int n_seqs, int T, const int* seq_slot, float* state,
                                long long state_ld, const SsdShape& s, cudaStream_t stream) {
  const int n = s.inner() / groups;
  auto movers = [&](int threads) { return s.taps > 1 ? (long long)n_seqs * ((s.channels() + threads - 1) / threads) : 0; };
  const bool four = n % 4 == 0 && ldy % 4 == 0 && ld % 4 == 0 && ((uintptr_t)y & 15) == 0 && ((uintptr_t)proj & 15) == 0 &&
                    ((uintptr_t)w & 15) == 0 && ((uintptr_t)out & 15) == 0;
  if (four && n <= 1024) {
    const long long norm_blocks = ((long long)T * groups + GN_WARPS - 1) / GN_WARPS, all = norm_blocks + movers(GN_WARPS * 32);
    if (all > 0x7fffffffLL) return DLGO_ERR_SIZE;
    const dim3 grid((unsigned)all), block(GN_WARPS * 32);
#define GN_ARGS grid, block, 0, stream, y, ldy, proj, ld, w, out, groups, eps, seqs, T, (int)norm_blocks, seq_slot, state, state_ld, s
    if (n <= 128) launch_kernel(ssd_gate_norm_warp_kernel<TO, 1>, GN_ARGS);
    else if (n <= 256) launch_kernel(ssd_gate_norm_warp_kernel<TO, 2>, GN_ARGS);
    else if (n <= 512) launch_kernel(ssd_gate_norm_warp_kernel<TO, 4>, GN_ARGS);
    else launch_kernel(ssd_gate_norm_warp_kernel<TO, 8>, GN_ARGS);
#undef GN_ARGS
    return launch_status();
  }
  const int stash = n * sizeof(float) <= 40 * 1024;
  const int threads = n >= 2048 ? 512 : (n >= 512 ? 256 : (n >= 128 ? 128 : 64));
  const long long norm_blocks = (long long)T * groups, all = norm_blocks + movers(threads);
  if (all > 0x7fffffffLL) return DLGO_ERR_SIZE;
  launch_kernel(ssd_gate_norm_kernel<TO>, dim3((unsigned)all), dim3(threads), stash ? n * sizeof(float) : 0, stream, y, ldy,
                proj, ld, w, out, groups, eps, seqs, (int)norm_blocks, seq_slot, state, state_ld, s, stash);
  return launch_status();
}

static bool ssd_shape_ok(const SsdShape& s) {
  return s.H > 0 && s.G > 0 && s.H % s.G == 0 && s.N > 0 && s.N <= 512 && s.P > 0 && s.taps > 0 && s.H <= 65535;
}

template <int RS>
static int launch_ssd_segments(const float* xbc, int ld, const float* steps, const float* D, const int* tiles, int n_tiles,
                               int direct, const int* seq_slot, float* state, long long state_ld, float* scratch,
                               float* out, int ldo, SsdShape s, int vec, cudaStream_t stream) {
  using TL = SsdTile<RS>;
  const dim3 grid(n_tiles, s.H, ssd_col_blocks<RS>(s.P)), block = ssd_block<RS>(s.P);
  const size_t smem = sizeof(float) * 2 * TL::CH * TL::ROW;
  float* seg = direct ? nullptr : scratch;
  float* dec = direct ? nullptr : scratch + (size_t)n_tiles * s.H * s.N * s.P;
  if (!direct) {
    launch_kernel(ssd_segments_kernel<RS, SSD_LOCAL>, grid, block, smem, stream, xbc, ld, steps, D, tiles, n_tiles,
                  seq_slot, state, state_ld, seg, dec, out, ldo, s, direct, vec);
    int st = launch_status();
    if (st != DLGO_OK) return st;
    st = launch_ssd_carry(tiles, n_tiles, seq_slot, state, state_ld, seg, dec, s, stream);
    if (st != DLGO_OK) return st;
  }
  launch_kernel(ssd_segments_kernel<RS, SSD_FULL>, grid, block, smem, stream, xbc, ld, steps, D, tiles, n_tiles, seq_slot,
                state, state_ld, seg, dec, out, ldo, s, direct, vec);
  return launch_status();
}

}  // namespace dlgo

using namespace dlgo;

template <typename TO>
static int launch_ssd_conv(const float* proj, int ld, const float* w_taps, const float* w_bias, const float* dt_bias,
                           const float* a_log, const int* tiles, int n_tiles, const int* token_seq, const int* seq_slot,
                           const float* state, long long state_ld, TO* out, int ldo, float* steps, int log_decay,
                           const SsdShape& s, cudaStream_t stream) {
  const int C = s.channels();
  const bool four = s.taps <= 4 && C % 4 == 0 && s.inner() % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 &&
                    ((uintptr_t)proj & 15) == 0 && ((uintptr_t)out & 15) == 0 && ((uintptr_t)w_taps & 15) == 0;
  const int w = four ? 4 : 1;
  const dim3 grid(n_tiles, (C + SC_THREADS * w - 1) / (SC_THREADS * w) + 1), block(SC_THREADS);
#define CONV_ARGS grid, block, 0, stream, proj, ld, w_taps, w_bias, dt_bias, a_log, tiles, token_seq, seq_slot, state, \
                  state_ld, out, ldo, steps, log_decay, s
  if (four && s.taps == 4) launch_kernel(ssd_conv_kernel<TO, 4, 4>, CONV_ARGS);
  else if (four && s.taps == 3) launch_kernel(ssd_conv_kernel<TO, 3, 4>, CONV_ARGS);
  else if (four && s.taps == 2) launch_kernel(ssd_conv_kernel<TO, 2, 4>, CONV_ARGS);
  else if (four && s.taps == 1) launch_kernel(ssd_conv_kernel<TO, 1, 4>, CONV_ARGS);
  else launch_kernel(ssd_conv_kernel<TO, 0, 1>, CONV_ARGS);
#undef CONV_ARGS
  return launch_status();
}

// proj [T, ld] fp32 with the columns [z | x | B | C | dt]; w_taps [C, taps], w_bias [C], dt_bias, a_log [H] fp32;
// tiles [n_tiles, 3] (sequence, first packed token, count); out [T, ldo >= C] in `dtype`: x | B | C; steps [T, H, 2] fp32:
// d and f, or with `log_decay` d and the logarithm of f
DLGO_EXPORT int dlgo_ssd_conv(const float* proj, int ld, const float* w_taps, const float* w_bias, const float* dt_bias,
                              const float* a_log, const int* tiles, int n_tiles, const int* token_seq,
                              const int* seq_slot, const float* state, long long state_ld, void* out, int dtype, int ldo,
                              float* steps, int log_decay, int H, int G, int N, int P, int taps, cudaStream_t stream) {
  if (n_tiles <= 0) return DLGO_OK;
  const SsdShape s{H, G, N, P, taps};
  if (!ssd_shape_ok(s)) return DLGO_ERR_SIZE;
#define CONV_ARGS(T) proj, ld, w_taps, w_bias, dt_bias, a_log, tiles, n_tiles, token_seq, seq_slot, state, state_ld, (T*)out, ldo, \
                     steps, log_decay, s, stream
  if (dtype == DLGO_F32) return launch_ssd_conv<float>(CONV_ARGS(float));
  if (dtype == DLGO_BF16) return launch_ssd_conv<__nv_bfloat16>(CONV_ARGS(__nv_bfloat16));
#undef CONV_ARGS
  return DLGO_ERR_DTYPE;
}

// xbc [T, ld] fp32 (x | B | C) and steps of dlgo_ssd_conv; D [H] fp32 or null (0); tiles [n_tiles, 3], a sequence's segments side by
// side in token order; out [T, ldo >= H P] fp32.  `direct`: one segment per sequence; else scratch holds
// n_tiles * H * (N P + 1) floats.
DLGO_EXPORT int dlgo_ssd_segments(const float* xbc, int ld, const float* steps, const float* D, const int* tiles,
                                  int n_tiles, int direct, const int* seq_slot, float* state, long long state_ld,
                                  float* scratch, float* out, int ldo, int H, int G, int N, int P, int taps,
                                  cudaStream_t stream) {
  if (n_tiles <= 0) return DLGO_OK;
  const SsdShape s{H, G, N, P, taps};
  if (!ssd_shape_ok(s) || n_tiles > 65535 || (!direct && scratch == nullptr)) return DLGO_ERR_SIZE;
  const int vec = ((N | P | ld) & 3) == 0 && (state_ld & 3) == 0 && ((uintptr_t)xbc & 15) == 0 &&
                  ((uintptr_t)state & 15) == 0 && ((uintptr_t)scratch & 15) == 0;
#define SSD_ARGS xbc, ld, steps, D, tiles, n_tiles, direct, seq_slot, state, state_ld, scratch, out, ldo, s, vec, stream
  switch (ssd_row_split(N)) {
    case 1: return launch_ssd_segments<1>(SSD_ARGS);
    case 2: return launch_ssd_segments<2>(SSD_ARGS);
    case 4: return launch_ssd_segments<4>(SSD_ARGS);
    case 8: return launch_ssd_segments<8>(SSD_ARGS);
    case 16: return launch_ssd_segments<16>(SSD_ARGS);
    default: return launch_ssd_segments<32>(SSD_ARGS);
  }
#undef SSD_ARGS
}

// One token per sequence (token t belongs to sequence t of the step).
DLGO_EXPORT int dlgo_ssd_step(const float* proj, int ld, const float* w_taps, const float* w_bias, const float* dt_bias,
                              const float* a_log, const float* D, const int* seq_slot, float* state, long long state_ld,
                              float* out, int ldo, int T, int H, int G, int N, int P, int taps, cudaStream_t stream) {
  if (T <= 0) return DLGO_OK;
  const SsdShape s{H, G, N, P, taps};
  if (!ssd_shape_ok(s)) return DLGO_ERR_SIZE;
  const int vec = ((N | P) & 3) == 0 && (state_ld & 3) == 0 && ((uintptr_t)state & 15) == 0;
#define STEP_LAUNCH(RS) \
  launch_kernel(ssd_step_kernel<RS>, dim3(T, H, ssd_col_blocks<RS>(P)), ssd_block<RS>(P), 0, stream, proj, ld, w_taps, w_bias, \
                dt_bias, a_log, D, seq_slot, state, state_ld, out, ldo, s, vec)
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

// y [T, ldy] fp32, proj as above (its z columns gate), w [H P] fp32, out [T, H P] in `dtype`; `groups` divides H P;
// seqs [n_seqs, 3] (sequence, first packed token, count): every sequence of the step
DLGO_EXPORT int dlgo_ssd_gate_norm(const float* y, int ldy, const float* proj, int ld, const float* w, void* out, int dtype,
                                   int groups, float eps, const int* seqs, int n_seqs, int T, const int* seq_slot,
                                   float* state, long long state_ld, int H, int G, int N, int P, int taps, cudaStream_t stream) {
  if (T <= 0) return DLGO_OK;
  const SsdShape s{H, G, N, P, taps};
  if (!ssd_shape_ok(s) || groups <= 0 || s.inner() % groups || groups > 65535) return DLGO_ERR_SIZE;
#define GN_ARGS(T_) y, ldy, proj, ld, w, (T_*)out, groups, eps, seqs, n_seqs, T, seq_slot, state, state_ld, s, stream
  if (dtype == DLGO_F32) return launch_ssd_gate_norm<float>(GN_ARGS(float));
  if (dtype == DLGO_BF16) return launch_ssd_gate_norm<__nv_bfloat16>(GN_ARGS(__nv_bfloat16));
#undef GN_ARGS
  return DLGO_ERR_DTYPE;
}
