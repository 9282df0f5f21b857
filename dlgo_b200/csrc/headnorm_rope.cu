// Per-head RMS norm of queries and keys, rotary positions computed from the position itself, and the
// append of this step's keys and values to the paged cache, in one pass over the fp32 result of the
// q|k (or q|k|v) projection.
//
// proj[T, ld] (fp32): Hq query heads, then Hkv key heads of `dk` numbers each, then (unless `v_from_k`) Hkv value
// heads of `dv`; in the cache and in q_out every head is `hd` numbers wide (hd >= dk, dv) with zeros behind its own,
// so that keys and values share one page shape.  `bias` (fp32, one number per column, may be null) is added first.
// With `v_from_k` the value of a position is its key as projected (with the bias, before norm and rotation); value
// heads of their own are kept times `v_scale`.
//
//   head norm (w_q / w_k not null):  u <- u / sqrt(mean(u^2) + eps) * w      (plain weight, per head; the mean runs
//   over the first `norm_dim` numbers of a head: a head may be laid out with trailing zeros)
//   rotation of the first `rot` numbers of a head: (u_i, u_{i + rot/2}) turns by a = pos * freq[i],
//   with a = float(pos) * freq[i] in fp32 and cos / sin of that fp32 angle.
//
// q goes to q_out[T, Hq * hd] in the run's type; k and v go to the page of the token's position:
// pages[page_table[slot][pos / PS]][kv_head][pos % PS][:].  `clear`: zeros are left in proj (a sum that
// the projection's K-slices add themselves into and that must be zero again for the next step).
// Everything is fp32 until the final store.
#include "common.cuh"

namespace dlgo {

// Set when a token's position had no page in the table (-1): the append is skipped.
__device__ int g_headnorm_rope_error = 0;

constexpr int HR_WARPS = 4;

template <typename T>
__global__ void __launch_bounds__(HR_WARPS * 32)
headnorm_rope_append_kernel(float* proj, int ld, const float* __restrict__ bias,
                            const float* __restrict__ w_q, const float* __restrict__ w_k, float eps,
                            const float* __restrict__ freq, int rot, const int* __restrict__ token_pos,
                            const int* __restrict__ token_seq, const int* __restrict__ seq_slot,
                            const int* __restrict__ page_table, int max_pages, T* kpages,
                            T* vpages, T* q_out, int T_tokens, int Hq, int Hkv, int dk,
                            int dv, int hd, int page_size, int v_from_k, int write_cache, int clear, int norm_dim,
                            float v_scale) {
  extern __shared__ float hr_smem[];
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int heads = Hq + Hkv + (v_from_k ? 0 : Hkv);
  const long long item = (long long)blockIdx.x * HR_WARPS + warp;
  if (item >= (long long)T_tokens * heads) return;
  const int t = (int)(item / heads), head = (int)(item - (long long)t * heads);
  float* u = hr_smem + (size_t)warp * hd;
  // the step's own inputs: in place before the step's first kernel starts
  const int pos = token_pos[t];
  const bool is_q = head < Hq, is_k = !is_q && head < Hq + Hkv;
  T* kdst = nullptr;
  T* vdst = nullptr;
  if (!is_q && write_cache) {
    const int slot = seq_slot[token_seq[t]];
    const int page = page_table[(size_t)slot * max_pages + pos / page_size];
    if (page < 0) {
      if (lane == 0) atomicExch(&g_headnorm_rope_error, 1);
    } else {
      const int kvh = is_k ? head - Hq : head - Hq - Hkv;
      const size_t base = (((size_t)page * Hkv + kvh) * page_size + (size_t)(pos % page_size)) * hd;
      kdst = kpages + base;
      vdst = vpages + base;
    }
  }
  const float* w = is_q ? w_q : (is_k ? w_k : nullptr);
  pdl_wait();
  const bool is_v = !is_q && !is_k;
  const int n = is_v ? dv : dk;                  // this head's own numbers
  const size_t col = is_v ? (size_t)(Hq + Hkv) * dk + (size_t)(head - Hq - Hkv) * dv : (size_t)head * dk;
  float* src = proj + (size_t)t * ld + col;
  float ss = 0.f;
  for (int i = lane; i < n; i += 32) {
    float x = src[i];
    if (bias != nullptr) x += bias[col + i];
    u[i] = x;
    ss += x * x;
    if (is_k && v_from_k && vdst != nullptr) vdst[i] = from_float<T>(x);
  }
  if (is_k && v_from_k && vdst != nullptr)
    for (int i = n + lane; i < hd; i += 32) vdst[i] = from_float<T>(0.f);
  if (clear)                     // (after every load of the row has been issued: a store right behind a load holds the loads up)
    for (int i = lane; i < n; i += 32) src[i] = 0.f;
  if (is_v) {                    // a value head of its own: stored as projected
    if (vdst != nullptr)
      for (int i = lane; i < hd; i += 32) vdst[i] = from_float<T>(i < n ? u[i] * v_scale : 0.f);
    return;
  }
  ss = warp_sum(ss);
  const float r = (w != nullptr) ? 1.0f / sqrtf(ss / (float)norm_dim + eps) : 1.0f;
  __syncwarp();
  T* dst = is_q ? q_out + (size_t)t * Hq * hd + (size_t)head * hd : kdst;
  if (dst == nullptr) return;
  const int rh = rot / 2;
  const float p = (float)pos;
  for (int i = lane; i < rh; i += 32) {
    float a = u[i] * r, b = u[i + rh] * r;
    if (w != nullptr) { a *= w[i]; b *= w[i + rh]; }
    float sn, cs;
    sincosf(p * freq[i], &sn, &cs);
    dst[i] = from_float<T>(a * cs - b * sn);
    dst[i + rh] = from_float<T>(b * cs + a * sn);
  }
  for (int i = rot + lane; i < hd; i += 32) {
    float a = 0.f;
    if (i < n) {
      a = u[i] * r;
      if (w != nullptr) a *= w[i];
    }
    dst[i] = from_float<T>(a);
  }
}

// The same with a block per token (q|k|v with norms and no bias, heads of a multiple of four numbers up to 128 NV): the
// angles' cosines and sines once per token, rows in 16-byte pieces, several heads of a warp in flight together.
constexpr int HT_WARPS = 8, HT_HEADS = 3;

__device__ __forceinline__ void ht_store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void ht_store2(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

template <typename T, int NV>
__global__ void __launch_bounds__(HT_WARPS * 32)
headnorm_rope_token_kernel(float* proj, int ld, const float* __restrict__ w_q, const float* __restrict__ w_k, float eps,
                           const float* __restrict__ freq, int rot, const int* __restrict__ token_pos,
                           const int* __restrict__ token_seq, const int* __restrict__ seq_slot,
                           const int* __restrict__ page_table, int max_pages, T* kpages, T* vpages, T* q_out, int Hq,
                           int Hkv, int dk, int dv, int hd, int page_size, int write_cache, int clear, float v_scale) {
  extern __shared__ __align__(16) float ht_smem[];
  pdl_launch_dependents();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, rh = rot / 2;
  float* cs = ht_smem;                                             // [rh] cosines, [rh] sines
  float* u_s = ht_smem + ((2 * rh + 3) & ~3) + warp * (128 * NV);  // a head, normed
  const int pos = token_pos[t];
  long long row_base = -1;
  if (write_cache) {
    const int page = page_table[(size_t)seq_slot[token_seq[t]] * max_pages + pos / page_size];
    if (page < 0) {
      if (threadIdx.x == 0) atomicExch(&g_headnorm_rope_error, 1);
    } else {
      row_base = ((long long)page * Hkv * page_size + pos % page_size) * hd;
    }
  }
  bool angles = false;
  pdl_wait();
  const int heads = Hq + 2 * Hkv;
  float* row = proj + (size_t)t * ld;
  for (int g = warp; g - warp < heads; g += HT_WARPS * HT_HEADS) {      // (every warp takes part in the first round)
    float4 x[HT_HEADS][NV];
#pragma unroll
    for (int k = 0; k < HT_HEADS; ++k) {
      const int head = g + k * HT_WARPS;
      const bool is_v = head >= Hq + Hkv;
      const int n = is_v ? dv : dk;
      float* src = row + (is_v ? (size_t)(Hq + Hkv) * dk + (size_t)(head - Hq - Hkv) * dv : (size_t)head * dk);
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int i = (v * 32 + lane) * 4;
        x[k][v] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (head < heads && i < n) x[k][v] = *reinterpret_cast<const float4*>(src + i);
      }
    }
    if (!angles) {                                                 // (while the first rows are on their way)
      for (int i = threadIdx.x; i < rh; i += HT_WARPS * 32) sincosf((float)pos * freq[i], &cs[rh + i], &cs[i]);
      __syncthreads();
      angles = true;
    }
#pragma unroll
    for (int k = 0; k < HT_HEADS; ++k) {
      const int head = g + k * HT_WARPS;
      if (head >= heads) break;
      const bool is_q = head < Hq, is_v = head >= Hq + Hkv;
      const int n = is_v ? dv : dk;
      if (clear) {
        float* src = row + (is_v ? (size_t)(Hq + Hkv) * dk + (size_t)(head - Hq - Hkv) * dv : (size_t)head * dk);
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          const int i = (v * 32 + lane) * 4;
          if (i < n) *reinterpret_cast<float4*>(src + i) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
      }
      T* dst = is_q ? q_out + ((size_t)t * Hq + head) * hd
                    : (row_base < 0 ? nullptr
                                    : (is_v ? vpages : kpages) + row_base + (size_t)(head - Hq - (is_v ? Hkv : 0)) * page_size * hd);
      float r = v_scale;
      const float* w = nullptr;
      if (!is_v) {
        float ss = 0.f;
#pragma unroll
        for (int v = 0; v < NV; ++v)
          ss += (x[k][v].x * x[k][v].x + x[k][v].y * x[k][v].y) + (x[k][v].z * x[k][v].z + x[k][v].w * x[k][v].w);
        r = 1.0f / sqrtf(warp_sum(ss) / (float)dk + eps);
        w = is_q ? w_q : w_k;
      }
      __syncwarp();                                                // the head before has been read
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int i = (v * 32 + lane) * 4;
        float4 o = make_float4(x[k][v].x * r, x[k][v].y * r, x[k][v].z * r, x[k][v].w * r);
        if (w != nullptr && i < n) {
          const float4 m = *reinterpret_cast<const float4*>(w + i);
          o.x *= m.x; o.y *= m.y; o.z *= m.z; o.w *= m.w;
        }
        *reinterpret_cast<float4*>(u_s + i) = o;                   // (zeros behind the head's own numbers)
      }
      __syncwarp();
      if (dst == nullptr) continue;
      const int turned = is_v ? 0 : rot;
      if ((rh & 1) == 0) {                                         // (then rot is a multiple of four: whole pieces)
        for (int i = 2 * lane; i < (turned >> 1); i += 64) {
          const float2 a = *reinterpret_cast<const float2*>(u_s + i), b = *reinterpret_cast<const float2*>(u_s + i + rh);
          const float2 c = *reinterpret_cast<const float2*>(cs + i), sn = *reinterpret_cast<const float2*>(cs + rh + i);
          ht_store2(dst + i, a.x * c.x - b.x * sn.x, a.y * c.y - b.y * sn.y);
          ht_store2(dst + i + rh, b.x * c.x + a.x * sn.x, b.y * c.y + a.y * sn.y);
        }
        for (int i = turned + 2 * lane; i < hd; i += 64) ht_store2(dst + i, u_s[i], u_s[i + 1]);
      } else {
        for (int i = lane; i < (turned >> 1); i += 32) {
          const float a = u_s[i], b = u_s[i + rh];
          dst[i] = from_float<T>(a * cs[i] - b * cs[rh + i]);
          dst[i + rh] = from_float<T>(b * cs[i] + a * cs[rh + i]);
        }
        for (int i = turned + lane; i < hd; i += 32) dst[i] = from_float<T>(u_s[i]);
      }
    }
  }
}

template <typename T>
int launch_headnorm_rope(float* proj, int ld, const float* bias, const float* w_q, const float* w_k, float eps,
                         const float* freq, int rot, const int* token_pos, const int* token_seq, const int* seq_slot,
                         const int* page_table, int max_pages, void* kpages, void* vpages, void* q_out, int T_tokens,
                         int Hq, int Hkv, int dk, int dv, int hd, int page_size, int v_from_k, int write_cache, int clear,
                         int norm_dim, float v_scale, cudaStream_t stream) {
  const int heads = Hq + Hkv + (v_from_k ? 0 : Hkv);
  const long long items = (long long)T_tokens * heads;
  const long long blocks = (items + HR_WARPS - 1) / HR_WARPS;
  if (blocks > 0x7fffffffLL) return DLGO_ERR_SIZE;
  const int wide = dk > dv ? dk : dv;
  if (!v_from_k && bias == nullptr && w_q != nullptr && w_k != nullptr && norm_dim == dk && ((dk | dv | ld) & 3) == 0 && hd % 2 == 0 && hd <= 256 &&
      (((uintptr_t)proj | (uintptr_t)w_q | (uintptr_t)w_k) & 15) == 0) {
    const int nv = (hd > wide ? hd : wide) <= 128 ? 1 : 2;
    const size_t ht = sizeof(float) * (((size_t)rot + 3) / 4 * 4 + HT_WARPS * 128 * nv);
#define HT_ARGS dim3(T_tokens), dim3(HT_WARPS * 32), ht, stream, proj, ld, w_q, w_k, eps, freq, rot, token_pos, token_seq, seq_slot, \
                page_table, max_pages, (T*)kpages, (T*)vpages, (T*)q_out, Hq, Hkv, dk, dv, hd, page_size, write_cache, clear, v_scale
    if (nv == 1) launch_kernel(headnorm_rope_token_kernel<T, 1>, HT_ARGS);
    else launch_kernel(headnorm_rope_token_kernel<T, 2>, HT_ARGS);
#undef HT_ARGS
    return launch_status();
  }
  const size_t smem = (size_t)HR_WARPS * hd * sizeof(float);
  if (smem > 48 * 1024) return DLGO_ERR_SIZE;
  launch_kernel(headnorm_rope_append_kernel<T>, dim3((unsigned)blocks), dim3(HR_WARPS * 32), smem, stream, proj, ld,
                bias, w_q, w_k, eps, freq, rot, token_pos, token_seq, seq_slot, page_table, max_pages, (T*)kpages,
                (T*)vpages, (T*)q_out, T_tokens, Hq, Hkv, dk, dv, hd, page_size, v_from_k, write_cache, clear, norm_dim, v_scale);
  return launch_status();
}

}  // namespace dlgo

DLGO_EXPORT int dlgo_headnorm_rope_append(float* proj, int ld, const float* bias, const float* w_q, const float* w_k,
                                          float eps, const float* freq, int rot, const int* token_pos,
                                          const int* token_seq, const int* seq_slot, const int* page_table,
                                          int max_pages, void* kpages, void* vpages, void* q_out, int dtype, int T,
                                          int Hq, int Hkv, int dk, int dv, int hd, int page_size, int v_from_k,
                                          int write_cache, int clear, int norm_dim, float v_scale, cudaStream_t stream) {
  if (T <= 0) return DLGO_OK;
  if (Hq <= 0 || Hkv <= 0 || dk <= 0 || dv <= 0 || hd < dk || hd < dv || rot < 0 || rot > dk || rot % 2)
    return DLGO_ERR_SIZE;
  if (v_from_k && dv != dk) return DLGO_ERR_SIZE;
  if (rot > 0 && freq == nullptr) return DLGO_ERR_SIZE;
  if (norm_dim <= 0 || norm_dim > dk) return DLGO_ERR_SIZE;
  if (ld < (Hq + Hkv) * dk + (v_from_k ? 0 : Hkv * dv)) return DLGO_ERR_SIZE;
  if (dtype == DLGO_F32)
    return dlgo::launch_headnorm_rope<float>(proj, ld, bias, w_q, w_k, eps, freq, rot, token_pos, token_seq, seq_slot,
                                             page_table, max_pages, kpages, vpages, q_out, T, Hq, Hkv, dk, dv, hd,
                                             page_size, v_from_k, write_cache, clear, norm_dim, v_scale, stream);
  if (dtype == DLGO_BF16)
    return dlgo::launch_headnorm_rope<__nv_bfloat16>(proj, ld, bias, w_q, w_k, eps, freq, rot, token_pos, token_seq,
                                                     seq_slot, page_table, max_pages, kpages, vpages, q_out, T, Hq,
                                                     Hkv, dk, dv, hd, page_size, v_from_k, write_cache, clear, norm_dim, v_scale, stream);
  return DLGO_ERR_DTYPE;
}

// The error word (1: a position had no page), cleared by the read.
DLGO_EXPORT int dlgo_headnorm_rope_error() {
  int v = 0, zero = 0;
  if (cudaMemcpyFromSymbol(&v, dlgo::g_headnorm_rope_error, sizeof(int)) != cudaSuccess) return -1;
  if (v) cudaMemcpyToSymbol(dlgo::g_headnorm_rope_error, &zero, sizeof(int));
  return v;
}
