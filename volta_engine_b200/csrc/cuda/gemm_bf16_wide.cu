// Prefill linear with bf16 weights and activations on 256 x 256 output tiles:   out[t, n] = sum_k W[n, k] * X[t, k]
//
// With one 128-feature tile per CTA (gemm_tcgen05.cu) every k step of 64 brings 48 KB from L2 for 2.1 MFLOP of tensor work, and
// the loop waits on L2. Here two 128-feature tiles share one 256-token activation tile: 64 KB for 4.2 MFLOP, two accumulators of
// 256 TMEM columns, three 64 KB stages. Warp roles (192 threads): warp 0 TMA producer, warp 1 TMEM owner + MMA issuer, warps
// 2..5 epilogue (TMEM lane = output feature, column = token). Rows and columns outside the matrices read as zero and are not
// stored; K need not be a multiple of 64. Every wait is bounded.
#include "common.cuh"
#include "gemm_epilogue.cuh"
#include "tmap.h"

namespace ve {

struct WideBf16Params {
  int N, T, K;
  float alpha;
  __nv_bfloat16* out;
  float* out_f32;
  long ldo;
  const __nv_bfloat16* residual;
  long ldr;
  int* status;
  const float* bias;
};

constexpr int WB_SUB = 128 * 128, WB_B = 256 * 128, WB_STAGE = 2 * WB_SUB + WB_B, WB_STAGES = 3;
constexpr int WB_SMEM = WB_STAGES * WB_STAGE + 1024;

__global__ void __launch_bounds__(192, 1)
gemm_bf16_wide_kernel(const WideBf16Params p, const __grid_constant__ CUtensorMap amap, const __grid_constant__ CUtensorMap bmap) {
  static_assert(WB_SMEM <= 227 * 1024, "shared memory budget");
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  __shared__ uint64_t full[WB_STAGES], empty[WB_STAGES], acc_full;
  __shared__ uint32_t tmem_holder;
  __shared__ int s_fail;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * 256, t0 = blockIdx.y * 256;
  const int nkt = (p.K + 63) / 64;
  if (threadIdx.x == 0) {
    for (int s = 0; s < WB_STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(&acc_full, 1);
    s_fail = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(&tmem_holder, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_holder;
  if (warp == 0) {
    if (elect_one()) {
      prefetch_tmap(&amap);
      prefetch_tmap(&bmap);
      for (int kt = 0; kt < nkt; ++kt) {
        const int s = kt % WB_STAGES;
        if (!mbar_wait(&empty[s], ((kt / WB_STAGES) & 1) ^ 1)) {
          atomicExch(&s_fail, 1);
          break;
        }
        uint8_t* st = smem + (size_t)s * WB_STAGE;         // [A0][A1][B]
        mbar_expect_tx(&full[s], WB_STAGE);
        tma_load_2d(st, &amap, &full[s], kt * 64, n0);
        tma_load_2d(st + WB_SUB, &amap, &full[s], kt * 64, n0 + 128);
        tma_load_2d(st + 2 * WB_SUB, &bmap, &full[s], kt * 64, t0);
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t idesc = make_idesc_f16(1, 1, 128, 256);
      bool ok = true;
      for (int kt = 0; kt < nkt && ok; ++kt) {
        const int s = kt % WB_STAGES;
        ok = mbar_wait(&full[s], (kt / WB_STAGES) & 1);
        if (!ok) break;
        tc_fence_after();
        const uint32_t st = smem_u32(smem + (size_t)s * WB_STAGE);
        const uint64_t bd = make_desc_sw128(st + 2 * WB_SUB);
#pragma unroll
        for (int sub = 0; sub < 2; ++sub) {
          const uint64_t ad = make_desc_sw128(st + sub * WB_SUB);
#pragma unroll
          for (int kb = 0; kb < 4; ++kb) tc_mma_f16(tmem_base + sub * 256, ad + kb * 2, bd + kb * 2, idesc, (kt | kb) ? 1u : 0u);
        }
        tc_commit(&empty[s]);
      }
      if (!ok) atomicExch(&s_fail, 1);
      tc_commit(&acc_full);
    }
  } else {
    const bool ok = mbar_wait(&acc_full, 0);
    if (!ok) atomicExch(&s_fail, 1);
    tc_fence_after();
    asm volatile("bar.sync 1, 128;" ::: "memory");        // one answer for the four warps: they meet at barriers below
    if (!*(volatile int*)&s_fail)
      for (int sub = 0; sub < 2; ++sub)
        if (n0 + sub * 128 < p.N)
          store_tile<256>(smem, tmem_base + sub * 256, warp & 3, (warp - 2) * 32 + lane, n0 + sub * 128, t0,
                          TileOut{p.N, p.T, p.alpha, p.out, p.out_f32, p.ldo, p.residual, p.ldr, p.bias});
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
  if (threadIdx.x == 0 && s_fail && p.status) atomicExch(p.status, (int)kErrMbarTimeout);
}

}  // namespace ve

using namespace ve;

extern "C" {

// Arguments as ve_gemm_bf16: W [N, K] (pitch ldw), X [T, K] (pitch ldx), pitches multiples of 8 elements; out bf16 or out_f32; bias fp32 [N] or null.
int ve_gemm_bf16_wide(const void* W, long ldw, const void* X, long ldx, void* out, long ldo, void* out_f32, const void* residual, long ldr, int T, int N,
                      int K, float alpha, const void* bias, void* status, cudaStream_t st) {
  if (T <= 0 || N <= 0) return 0;
  if (K < 1) return cudaErrorInvalidValue;
  CUtensorMap amap, bmap;
  int rc = make_tmap_2d(&amap, W, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, N, K, (uint64_t)ldw * 2, 128, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  rc = make_tmap_2d(&bmap, X, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, T, K, (uint64_t)ldx * 2, 256, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(gemm_bf16_wide_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, WB_SMEM);
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  WideBf16Params p{N, T, K, alpha, (__nv_bfloat16*)out, (float*)out_f32, ldo, (const __nv_bfloat16*)residual, ldr, (int*)status, (const float*)bias};
  gemm_bf16_wide_kernel<<<dim3((N + 255) / 256, (T + 255) / 256), 192, WB_SMEM, st>>>(p, amap, bmap);
  return (int)cudaGetLastError();
}

}  // extern "C"
