// Output tile of a GEMM whose TMEM lanes are output features and whose columns are tokens: TMEM -> shared memory (one row of 128
// features per token, padded by 16 bytes) -> global memory in 16-byte pieces of whole rows. Storing straight from the TMEM layout
// writes 64 bytes per warp and token; that took 25 us per 128 x 256 tile whatever K was.
#pragma once
#include "common.cuh"

namespace ve {

struct TileOut {
  int N, t_end;                     // features of the matrix, end of the tile's valid tokens
  float alpha;
  __nv_bfloat16* out;               // or out_f32
  float* out_f32;
  long ldo;
  const __nv_bfloat16* residual;    // optional, added before rounding
  long ldr;
  const float* bias;                // optional [N], added before rounding
};

// Called by four warps (etid 0..127, `quarter` = the TMEM lane quarter of the calling warp) once the accumulator is complete and the
// staging memory (COLS * 528 bytes) is free. n0: feature of lane 0; t0: token of column 0. Ends with a barrier of the 128 threads.
template <int COLS>
VE_DEVINL void store_tile(uint8_t* stage, uint32_t tmem, int quarter, int etid, int n0, int t0, const TileOut& o) {
  const int lane = etid & 31, col = quarter * 32 + lane;
  const int rows = min(COLS, o.t_end - t0);
  const uint32_t lane_addr = tmem + ((uint32_t)(quarter * 32) << 16);
  const float b = o.bias && n0 + col < o.N ? o.bias[n0 + col] : 0.f;
#pragma unroll 1
  for (int c0 = 0; c0 < rows; c0 += 16) {
    uint32_t r[16];
    tmem_ld16(lane_addr + c0, r);
    tmem_ld_wait();
    if (o.out_f32) {
#pragma unroll
      for (int j = 0; j < 16; ++j) reinterpret_cast<float*>(stage + (c0 + j) * 528)[col] = fmaf(__uint_as_float(r[j]), o.alpha, b);
    } else if (o.residual) {          // the sum is rounded once: keep the product in fp32 until the residual is added
#pragma unroll
      for (int j = 0; j < 16; ++j) reinterpret_cast<float*>(stage + (c0 + j) * 528)[col] = fmaf(__uint_as_float(r[j]), o.alpha, b);
    } else {
#pragma unroll
      for (int j = 0; j < 16; ++j) reinterpret_cast<__nv_bfloat16*>(stage + (c0 + j) * 272)[col] = f2bf(fmaf(__uint_as_float(r[j]), o.alpha, b));
    }
  }
  asm volatile("bar.sync 1, 128;" ::: "memory");
  const int live = min(128, o.N - n0);
  if (o.out_f32) {
    const bool vec = !((uintptr_t)o.out_f32 & 15) && o.ldo % 4 == 0;
    for (int i = etid; i < rows * 32; i += 128) {
      const int r = i >> 5, c = (i & 31) * 4;
      const float4 v = *reinterpret_cast<const float4*>(stage + r * 528 + c * 4);
      float* dst = o.out_f32 + (long)(t0 + r) * o.ldo + n0 + c;
      if (vec && c + 4 <= live) *reinterpret_cast<float4*>(dst) = v;
      else {
        const float f[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (c + e < live) dst[e] = f[e];
      }
    }
  } else if (o.residual) {
    const bool vec = !((uintptr_t)o.out & 7) && o.ldo % 4 == 0 && !((uintptr_t)o.residual & 7) && o.ldr % 4 == 0;
    for (int i = etid; i < rows * 32; i += 128) {
      const int r = i >> 5, c = (i & 31) * 4;
      const float4 v = *reinterpret_cast<const float4*>(stage + r * 528 + c * 4);
      __nv_bfloat16* dst = o.out + (long)(t0 + r) * o.ldo + n0 + c;
      const __nv_bfloat16* res = o.residual + (long)(t0 + r) * o.ldr + n0 + c;
      if (vec && c + 4 <= live) {
        const uint2 b = *reinterpret_cast<const uint2*>(res);
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x + __uint_as_float(b.x << 16), v.y + __uint_as_float(b.x & 0xffff0000u));
        const __nv_bfloat162 hi = __floats2bfloat162_rn(v.z + __uint_as_float(b.y << 16), v.w + __uint_as_float(b.y & 0xffff0000u));
        *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
      } else {
        const float f[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (c + e < live) dst[e] = f2bf(f[e] + bf2f(res[e]));
      }
    }
  } else {
    const bool vec = !((uintptr_t)o.out & 15) && o.ldo % 8 == 0;
    for (int i = etid; i < rows * 16; i += 128) {
      const int r = i >> 4, c = (i & 15) * 8;
      const uint4 v = *reinterpret_cast<const uint4*>(stage + r * 272 + c * 2);
      __nv_bfloat16* dst = o.out + (long)(t0 + r) * o.ldo + n0 + c;
      if (vec && c + 8 <= live) *reinterpret_cast<uint4*>(dst) = v;
      else {
        const __nv_bfloat16* f = reinterpret_cast<const __nv_bfloat16*>(&v);
#pragma unroll
        for (int e = 0; e < 8; ++e)
          if (c + e < live) dst[e] = f[e];
      }
    }
  }
  asm volatile("bar.sync 1, 128;" ::: "memory");
}

}  // namespace ve
