// The gates of the real-gated linear recurrent unit (rglru.cu) for prompts in bfloat16, on the tensor cores (tcgen05),
// with what follows them up to a segment's end in the epilogue.
//
// A part of B channels has two matrices [B, B] (r, i), its rows of u are [T, B] (the parts one after another).  The
// WEIGHT is the M operand (128 output channels of one part), 32 tokens are N, so an accumulator's lane is a channel and
// its columns are the tokens of one segment in order: the thread that owns the lane forms a_t and the input of every
// token and walks the recurrence from zero in its registers.
//
//   z[t, part, 0 .. B) = a_t,  z[t, part, B .. 2 B) = sqrt(1 - a_t^2) i_t u_t;  per segment: its end, sum of log a_t
//
// A CTA keeps its 128 rows of both matrices in shared memory for good and walks segments (a few CTAs per block of
// channels); the segments' rows of u arrive by TMA (128-byte swizzle, no multicast) in four stages; four accumulator
// pairs in tensor memory, each with four epilogue warps of its own, so that segments' elementwise work runs beside one
// another's and the next products.  Warp 0 loads, warp 1 issues MMAs, the others are the epilogues.  Every wait is bounded
// and sets an error word.
#include "common.cuh"
#include "tcgen05.cuh"

namespace dlgo {

using namespace sm100;

constexpr int GU_TOK = 32, GU_M = 128, GU_K = 64, GU_GROUPS = 4, GU_THREADS = 64 + GU_GROUPS * 128;
constexpr int GU_W_BYTES = GU_M * GU_K * 2, GU_U_BYTES = GU_TOK * GU_K * 2;      // of one k-block
constexpr int GU_TMEM = GU_GROUPS * 2 * GU_TOK;      // columns: a pair of 32 per group

__device__ int g_rglru_tc_error = 0;

struct GuParams {
  const __nv_bfloat16* u;       // [parts, T, B]
  const float* br;              // [W]
  const float* bi;
  const float* lam;
  const int* tiles;             // [n_tiles, 3]: segments of at most 32 tokens
  int n_tiles, T, W, B, parts, chunks;
  float rate;
  float* z;                     // [T, parts, 2 B]
  float* seg;                   // [n_tiles, 3, W]: end from zero, sum of the logarithms, (start: not written here)
};

__device__ __forceinline__ float gu_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gu_sigmoid(float x) { return gu_rcp(1.0f + __expf(-x)); }
// sqrt(1 - exp(2 x)) for x <= 0; near zero from the exponential's series, whose terms do not cancel
__device__ __forceinline__ float gu_input_factor(float x, float a) {
  const float y = 2.0f * x;
  float s = fmaf(y, 1.0f / 40320.0f, 1.0f / 5040.0f);
  s = fmaf(y, s, 1.0f / 720.0f);
  s = fmaf(y, s, 1.0f / 120.0f);
  s = fmaf(y, s, 1.0f / 24.0f);
  s = fmaf(y, s, 1.0f / 6.0f);
  s = fmaf(y, s, 0.5f);
  s = -y * fmaf(y, s, 1.0f);
  const float v = y > -0.5f ? s : fmaf(-a, a, 1.0f);
  float r;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}

__global__ void __launch_bounds__(GU_THREADS, 1)
rglru_gates_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_u,
                      const __grid_constant__ GuParams p) {
  extern __shared__ uint8_t gu_smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)gu_smem_raw + 1023) & ~(uintptr_t)1023);
  const int nk = (p.B + GU_K - 1) / GU_K;
  uint8_t* w_s = smem;                                   // [nk][r: 128 rows | i: 128 rows]
  uint8_t* u_s = w_s + nk * 2 * GU_W_BYTES;              // [groups][nk][32 rows]
  uint64_t* w_full = (uint64_t*)(u_s + GU_GROUPS * nk * GU_U_BYTES);
  uint64_t* u_full = w_full + 1;                         // [groups], like the next three
  uint64_t* u_empty = u_full + GU_GROUPS;
  uint64_t* acc_full = u_empty + GU_GROUPS;
  uint64_t* acc_empty = acc_full + GU_GROUPS;
  uint32_t* tmem_slot = (uint32_t*)(acc_empty + GU_GROUPS);
  volatile int* abort_flag = (volatile int*)(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int part = blockIdx.y / p.chunks, c0 = (blockIdx.y - part * p.chunks) * GU_M;
  if (threadIdx.x == 0) {
    mbar_init(w_full, 1);
    for (int b = 0; b < GU_GROUPS; ++b) {
      mbar_init(&u_full[b], 1);
      mbar_init(&u_empty[b], 1);
      mbar_init(&acc_full[b], 1);
      mbar_init(&acc_empty[b], 4);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&map_w);
    tma_prefetch_desc(&map_u);
  }
  __syncthreads();
  if (warp == 0 && elect_one()) {                        // weights: nothing of the step writes them
    mbar_expect_tx(w_full, nk * 2 * GU_W_BYTES);
    for (int kb = 0; kb < nk; ++kb) {
      tma_load_2d(w_s + kb * 2 * GU_W_BYTES, &map_w, w_full, kb * GU_K, part * 2 * p.B + c0);
      tma_load_2d(w_s + kb * 2 * GU_W_BYTES + GU_W_BYTES, &map_w, w_full, kb * GU_K, part * 2 * p.B + p.B + c0);
    }
  }
  pdl_wait();
  if (warp == 1) {
    tmem_alloc(tmem_slot, GU_TMEM);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;
  // (only now: a tensor-core kernel behind this one allocates tensor memory in its prologue)
  pdl_launch_dependents();

  if (warp == 0) {
    if (elect_one()) {
      int it = 0;
      for (int tile = blockIdx.x; tile < p.n_tiles; tile += gridDim.x, ++it) {
        const int s = it % GU_GROUPS;
        if (it >= GU_GROUPS && !mbar_wait(&u_empty[s], (it / GU_GROUPS - 1) & 1, abort_flag)) break;
        mbar_expect_tx(&u_full[s], nk * GU_U_BYTES);
        const int row = part * p.T + p.tiles[3 * tile + 1];
        for (int kb = 0; kb < nk; ++kb)
          tma_load_2d(u_s + (s * nk + kb) * GU_U_BYTES, &map_u, &u_full[s], kb * GU_K, row);
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t idesc = umma_idesc_bf16(GU_M, GU_TOK);
      bool ok = mbar_wait(w_full, 0, abort_flag);
      int it = 0;
      for (int tile = blockIdx.x; ok && tile < p.n_tiles; tile += gridDim.x, ++it) {
        const int s = it % GU_GROUPS;
        if (it >= GU_GROUPS) ok = mbar_wait(&acc_empty[s], (it / GU_GROUPS - 1) & 1, abort_flag);
        if (ok) ok = mbar_wait(&u_full[s], (it / GU_GROUPS) & 1, abort_flag);
        if (!ok) break;
        tc_fence_after_sync();
        const uint32_t w_addr = smem_u32(w_s), u_addr = smem_u32(u_s + s * nk * GU_U_BYTES);
        const uint32_t d = tmem_base + (uint32_t)(s * 2 * GU_TOK);
        for (int kb = 0; kb < nk; ++kb) {
          const uint64_t dr = umma_desc_k_sw128(w_addr + kb * 2 * GU_W_BYTES);
          const uint64_t di = umma_desc_k_sw128(w_addr + kb * 2 * GU_W_BYTES + GU_W_BYTES);
          const uint64_t du = umma_desc_k_sw128(u_addr + kb * GU_U_BYTES);
#pragma unroll
          for (int k = 0; k < GU_K / 16; ++k) {
            umma_bf16(d, dr + 2 * k, du + 2 * k, idesc, (kb | k) != 0);
            umma_bf16(d + GU_TOK, di + 2 * k, du + 2 * k, idesc, (kb | k) != 0);
          }
        }
        umma_commit(&u_empty[s]);
        umma_commit(&acc_full[s]);
      }
    }
  } else {
    const int group = (warp - 2) >> 2, quarter = warp & 3;       // (a warp reads the tensor-memory lanes of its quarter)
    const int cb = c0 + quarter * 32 + lane;                     // channel of the part
    const bool mine = cb < p.B;
    const int c = part * p.B + (mine ? cb : 0);
    const float b_r = p.br[c], b_i = p.bi[c], lam = p.lam[c];
    const float rate_sp = p.rate * (fmaxf(lam, 0.f) + log1pf(expf(-fabsf(lam))));
    const size_t ldz = (size_t)2 * p.W;
    float* zc = p.z + (size_t)part * 2 * p.B + (mine ? cb : 0);
    int it = group;
    for (int tile = blockIdx.x + group * gridDim.x; tile < p.n_tiles; tile += GU_GROUPS * gridDim.x, it += GU_GROUPS) {
      const int t0 = p.tiles[3 * tile + 1], n = p.tiles[3 * tile + 2];
      __nv_bfloat16 uu[GU_TOK];
      const __nv_bfloat16* ur = p.u + ((size_t)part * p.T + t0) * p.B + (mine ? cb : 0);
#pragma unroll
      for (int q = 0; q < GU_TOK; ++q) uu[q] = ur[(size_t)min(q, n - 1) * p.B];      // on its way during the products
      if (!mbar_wait(&acc_full[group], (it / GU_GROUPS) & 1, abort_flag)) break;
      __syncwarp();                                              // (tensor-memory reads are the whole warp's)
      tc_fence_after_sync();
      float S = 0.f, total = 0.f;
      float* zt = zc + (size_t)t0 * ldz;
      const uint32_t taddr = tmem_base + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(group * 2 * GU_TOK);
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float r[GU_TOK / 2], i[GU_TOK / 2];
        tmem_ld_32x16(taddr + half * (GU_TOK / 2), r);
        tmem_ld_32x16(taddr + GU_TOK + half * (GU_TOK / 2), i);
        tmem_ld_wait();
        if (half == 1) {
          tc_fence_before_sync();
          __syncwarp();
          if (lane == 0) mbar_arrive(&acc_empty[group]);
        }
#pragma unroll
        for (int k = 0; k < GU_TOK / 2; ++k) {
          const int q = half * (GU_TOK / 2) + k;
          if (mine && q < n) {
            const float log_a = -rate_sp * gu_sigmoid(r[k] + b_r), a = __expf(log_a);
            const float in = gu_input_factor(log_a, a) * gu_sigmoid(i[k] + b_i) * __bfloat162float(uu[q]);
            zt[(size_t)q * ldz] = a;
            zt[(size_t)q * ldz + p.B] = in;
            total += log_a;
            S = fmaf(a, S, in);
          }
        }
        __syncwarp();
      }
      if (mine) {
        float* sg = p.seg + (size_t)tile * 3 * p.W + c;
        sg[0] = S;
        sg[p.W] = total;
      }
      __syncwarp();
    }
  }

  tc_fence_before_sync();
  __syncthreads();
  if (*abort_flag) {
    if (threadIdx.x == 0) atomicExch(&g_rglru_tc_error, 1);
    // give tile loads that may still be in flight time to land before shared memory is handed on
    for (int k = 0; k < 1000; ++k) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, GU_TMEM);
  }
}

namespace {

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiledFn encode_fn() {
  static EncodeTiledFn fn = nullptr;
  if (fn == nullptr) {
    void* q = nullptr;
    cudaDriverEntryPointQueryResult res;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &q, cudaEnableDefault, &res) == cudaSuccess &&
        res == cudaDriverEntryPointSuccess)
      fn = (EncodeTiledFn)q;
  }
  return fn;
}

int make_map(CUtensorMap* m, const void* base, long long rows, int K, int box_rows) {
  EncodeTiledFn fn = encode_fn();
  if (fn == nullptr) return DLGO_ERR_DRIVER;
  if (((uintptr_t)base & 15) != 0 || (K % 8) != 0) return DLGO_ERR_ALIGN;
  cuuint64_t dims[2] = {(cuuint64_t)K, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)K * 2};
  cuuint32_t box[2] = {(cuuint32_t)GU_K, (cuuint32_t)box_rows};
  cuuint32_t estr[2] = {1, 1};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? DLGO_OK : DLGO_ERR_DRIVER;
}

int smem_bytes(int B) {
  const int nk = (B + GU_K - 1) / GU_K;
  return nk * (2 * GU_W_BYTES + GU_GROUPS * GU_U_BYTES) + 1024 + 256;
}

}  // namespace
}  // namespace dlgo

using namespace dlgo;

// 1 if the kernel takes parts of B channels: rows in whole 16-byte pieces, both matrices' rows and four stages of u in
// shared memory
DLGO_EXPORT int dlgo_rglru_gates_tc_takes(int B) { return B > 0 && B % 8 == 0 && smem_bytes(B) <= 227 * 1024; }
DLGO_EXPORT int dlgo_rglru_gates_tc_tokens() { return GU_TOK; }

// u [parts, T, B] bf16, w [parts, 2 B, B] bf16 (rows of r, then of i), br, bi, lam [parts * B] fp32; tiles [n_tiles, 3]
// (sequence, first packed token, count <= 32); z [T, parts, 2 B], seg [n_tiles, 3, parts * B] fp32
DLGO_EXPORT int dlgo_rglru_gates_tc(const void* u, const void* w, const float* br, const float* bi, const float* lam,
                                    const int* tiles, int n_tiles, int T, int parts, int B, float rate, float* z, float* seg,
                                    cudaStream_t stream) {
  if (n_tiles <= 0 || T <= 0) return DLGO_OK;
  if (parts <= 0 || !dlgo_rglru_gates_tc_takes(B)) return DLGO_ERR_SIZE;
  CUtensorMap mw, mu;
  int st = make_map(&mw, w, (long long)parts * 2 * B, B, GU_M);
  if (st != DLGO_OK) return st;
  st = make_map(&mu, u, (long long)parts * T, B, GU_TOK);
  if (st != DLGO_OK) return st;
  static int sms = 0;
  if (sms == 0) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    cudaError_t e = cudaFuncSetAttribute(rglru_gates_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) { sms = 0; return (int)e; }
  }
  const int chunks = (B + GU_M - 1) / GU_M, smem = smem_bytes(B);
  int per_chunk = sms / (parts * chunks);                // (one CTA per SM: its threads' registers)
  if (per_chunk > (n_tiles + GU_GROUPS - 1) / GU_GROUPS) per_chunk = (n_tiles + GU_GROUPS - 1) / GU_GROUPS;
  if (per_chunk < 1) per_chunk = 1;
  if ((long long)parts * chunks > 65535) return DLGO_ERR_SIZE;
  GuParams p{(const __nv_bfloat16*)u, br, bi, lam, tiles, n_tiles, T, parts * B, B, parts, chunks, rate, z, seg};
  launch_kernel(rglru_gates_tc_kernel, dim3(per_chunk, parts * chunks), dim3(GU_THREADS), (size_t)smem, stream, mw, mu, p);
  return launch_status();
}

// The error word (1: a bounded wait ran out), cleared by the read.
DLGO_EXPORT int dlgo_rglru_gates_tc_error() {
  int v = 0, zero = 0;
  if (cudaMemcpyFromSymbol(&v, dlgo::g_rglru_tc_error, sizeof(int)) != cudaSuccess) return -1;
  if (v) cudaMemcpyToSymbol(dlgo::g_rglru_tc_error, &zero, sizeof(int));
  return v;
}
