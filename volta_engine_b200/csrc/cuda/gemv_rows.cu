// bf16 linears on a few rows (decode / verify steps), with the step in front in the prologue and the step behind in the
// epilogue, for decoders with an fp32 residual stream:
//   y[m][n] = sum_k W[n][k] x[m][k],   m < 16
//   prologue   0  x given in bf16
//              1  x = tanh(alpha h) w + b of the fp32 residual h
//              2  x = RMS norm over groups of columns of an fp32 row [* sigmoid(gate)]
//              3  x = PolyNorm of an fp32 row
//   epilogue   store fp32 or bf16, or h += scale * y on the fp32 residual
// The rows are the M side (16) of mma.sync.m16n8k16 and eight weight rows the N side. The order of k inside a product does
// not matter, so a lane takes eight consecutive k of one weight row with one 16-byte load and uses them as the B operands of
// two MMAs, the matching activations as the A operands: weights go from global memory to registers and are read once. The
// first weights are requested before the programmatic dependency wait, so they arrive while the kernel in front finishes.
// gemm_f32 is the plain fp32 product of the all-32-bit form.
#include "rowmath.cuh"

namespace ve {

struct RowsArgs {
  const __nv_bfloat16* W; long ldw;
  int N, K, M;                      // K: columns of W (a multiple of 8)
  int pro, kx;                      // kx <= K: columns of x (the rest read as zero)
  const void* x; long ldx;
  const float* w; const float* b; float alpha;
  int G, wlen;
  const float* gate; long ldg;
  const float* coef; float eps;
  float* out_f32; __nv_bfloat16* out; long ldo;
  float* h; long ldh; const float* scale;
  int pitch;                        // bytes per activation row in shared memory (prologue forms)
};

VE_DEVINL void rows_mma(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// Activations of the prologue forms -> bf16 rows in shared memory.
VE_DEVINL void rows_prologue(const RowsArgs& a, uint8_t* xs, float* red) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, K32 = (a.K + 31) / 32 * 32;
  const float* src = reinterpret_cast<const float*>(a.x);
  auto put = [&](int m, int k, float v) { reinterpret_cast<__nv_bfloat16*>(xs + m * a.pitch)[k] = f2bf(v); };
  for (int i = a.kx + tid; i < K32; i += 256)
    for (int m = 0; m < a.M; ++m) put(m, i, 0.f);
  if (a.pro == 1) {
    for (int k = tid; k < a.kx; k += 256) {
      const float wk = a.w[k], bk = a.b[k];
      for (int m = 0; m < a.M; ++m) put(m, k, dyt_of(src[m * a.ldx + k], a.alpha, wk, bk));
    }
  } else if (a.pro == 2) {
    const int groups = a.kx / a.G;
    if (groups * a.M >= 8) {
      for (int p = warp; p < groups * a.M; p += 8) {
        const int m = p / groups, c0 = (p % groups) * a.G;
        float ss = 0.f;
        for (int i = lane; i < a.G; i += 32) {
          const float v = src[m * a.ldx + c0 + i];
          ss = fmaf(v, v, ss);
        }
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)a.G + a.eps);
        for (int i = lane; i < a.G; i += 32) {
          const int c = c0 + i;
          float v = src[m * a.ldx + c] * inv * a.w[c % a.wlen];
          if (a.gate) v *= sigmoid_of(a.gate[m * a.ldg + c]);
          put(m, c, v);
        }
      }
    } else {
      for (int p = 0; p < groups * a.M; ++p) {
        const int m = p / groups, c0 = (p % groups) * a.G;
        float ss = 0.f;
        for (int i = tid; i < a.G; i += 256) {
          const float v = src[m * a.ldx + c0 + i];
          ss = fmaf(v, v, ss);
        }
        const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)a.G + a.eps);
        for (int i = tid; i < a.G; i += 256) {
          const int c = c0 + i;
          float v = src[m * a.ldx + c] * inv * a.w[c % a.wlen];
          if (a.gate) v *= sigmoid_of(a.gate[m * a.ldg + c]);
          put(m, c, v);
        }
      }
    }
  } else {
    for (int m = 0; m < a.M; ++m) {
      float s1 = 0.f, s2 = 0.f, s3 = 0.f;
      for (int i = tid; i < a.kx; i += 256) poly_sums(src[m * a.ldx + i], s1, s2, s3);
      s1 = block_sum(s1, red);
      s2 = block_sum(s2, red);
      s3 = block_sum(s3, red);
      const PolyScale ps = poly_scale(s1, s2, s3, a.kx, a.eps, a.coef);
      for (int i = tid; i < a.kx; i += 256) put(m, i, poly_of(src[m * a.ldx + i], ps));
    }
  }
  __syncthreads();
}

// 8 warps: R tiles of 8 weight rows x KS slices of k. Units of 32 k; slice s takes units s, s + KS, ...
template <int KS, bool FUSED>
__global__ void __launch_bounds__(256, 2) gemv_rows_kernel(const RowsArgs a) {
  constexpr int R = 8 / KS, PF = 8;
  extern __shared__ __align__(16) uint8_t xs[];
  __shared__ float part[8][16][8], red[33];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int ks = warp % KS, rt = warp / KS, n0 = (blockIdx.x * R + rt) * 8;
  const int units = (a.K + 31) / 32, mine = units > ks ? (units - ks + KS - 1) / KS : 0;
  const __nv_bfloat16* wr = a.W + (long)min(n0 + g, a.N - 1) * a.ldw + t * 8;
  auto load_w = [&](int j) -> uint4 {
    const int k = (ks + j * KS) * 32 + t * 8;
    if (j < mine && k < a.K) return __ldcs(reinterpret_cast<const uint4*>(wr + (k - t * 8)));
    return make_uint4(0, 0, 0, 0);
  };
  uint4 cur[PF];
#pragma unroll
  for (int j = 0; j < PF; ++j) cur[j] = load_w(j);
  grid_dep_wait();
  grid_dep_launch();
  if (FUSED) rows_prologue(a, xs, red);
  const __nv_bfloat16* xg = reinterpret_cast<const __nv_bfloat16*>(a.x);
  auto load_x = [&](int m, int k) -> uint4 {
    if (m >= a.M || k >= a.K) return make_uint4(0, 0, 0, 0);
    if (FUSED) return *reinterpret_cast<const uint4*>(xs + m * a.pitch + k * 2);
    return *reinterpret_cast<const uint4*>(xg + m * a.ldx + k);
  };
  float c[4] = {0.f, 0.f, 0.f, 0.f};
  for (int j0 = 0; j0 < mine; j0 += PF) {
    uint4 nxt[PF];
#pragma unroll
    for (int j = 0; j < PF; ++j) nxt[j] = load_w(j0 + PF + j);
#pragma unroll
    for (int j = 0; j < PF; ++j) {
      if (j0 + j < mine) {
        const int k = (ks + (j0 + j) * KS) * 32 + t * 8;
        const uint4 lo = load_x(g, k), hi = FUSED ? make_uint4(0, 0, 0, 0) : load_x(g + 8, k);     // fused rows: M <= 8
        rows_mma(c, lo.x, hi.x, lo.y, hi.y, cur[j].x, cur[j].y);
        rows_mma(c, lo.z, hi.z, lo.w, hi.w, cur[j].z, cur[j].w);
      }
    }
#pragma unroll
    for (int j = 0; j < PF; ++j) cur[j] = nxt[j];
  }
  part[warp][g][2 * t] = c[0];
  part[warp][g][2 * t + 1] = c[1];
  part[warp][g + 8][2 * t] = c[2];
  part[warp][g + 8][2 * t + 1] = c[3];
  __syncthreads();
  for (int i = tid; i < a.M * R * 8; i += 256) {
    const int m = i / (R * 8), q = i % (R * 8), r = q / 8, e = q % 8, n = (blockIdx.x * R + r) * 8 + e;
    if (n >= a.N) continue;
    float v = 0.f;
#pragma unroll
    for (int s = 0; s < KS; ++s) v += part[r * KS + s][m][e];
    if (a.h) a.h[m * a.ldh + n] = fmaf(v, a.scale ? a.scale[n] : 1.f, a.h[m * a.ldh + n]);
    else if (a.out_f32) a.out_f32[m * a.ldo + n] = v;
    else a.out[m * a.ldo + n] = f2bf(v);
  }
}

// out[t][n] = sum_k W[n][k] x[t][k], fp32 throughout. 64 x 64 tiles, 16 k per step, 4 x 4 outputs per thread.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ W, long ldw, const float* __restrict__ x, long ldx, float* __restrict__ out,
                                                       long ldo, int T, int N, int K) {
  __shared__ float sw[16][65], sx[16][65];
  const int tid = threadIdx.x, n0 = blockIdx.x * 64, t0 = blockIdx.y * 64, tn = (tid & 15) * 4, tt = (tid >> 4) * 4;
  grid_dep_wait();
  grid_dep_launch();
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = tid; i < 64 * 16; i += 256) {
      const int r = i >> 4, k = i & 15;
      sw[k][r] = (n0 + r < N && k0 + k < K) ? W[(long)(n0 + r) * ldw + k0 + k] : 0.f;
      sx[k][r] = (t0 + r < T && k0 + k < K) ? x[(long)(t0 + r) * ldx + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(sx[k][tt + i], sw[k][tn + j], acc[i][j]);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (t0 + tt + i < T && n0 + tn + j < N) out[(long)(t0 + tt + i) * ldo + n0 + tn + j] = acc[i][j];
}

template <int KS, bool FUSED>
static int launch_rows(const RowsArgs& a, cudaStream_t st) {
  const int smem = FUSED ? a.M * a.pitch : 0;
  static int attr = 0;
  if (smem > attr) {
    cudaError_t e = cudaFuncSetAttribute(gemv_rows_kernel<KS, FUSED>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
    attr = smem;
  }
  const int tiles = (a.N + 7) / 8;
  launch_pdl(gemv_rows_kernel<KS, FUSED>, dim3((tiles + 8 / KS - 1) / (8 / KS)), dim3(256), smem, st, a);
  return (int)cudaGetLastError();
}

}  // namespace ve

using namespace ve;

extern "C" {

// pro 0: x bf16 [M, K], M <= 16. pro 1..3: x fp32 [M, kx], M <= 8 and the activation rows fit in shared memory (else refused).
// Exactly one of h, out_f32 and out is written.
int ve_gemv_rows(const void* W, long ldw, int N, int K, int M, int pro, int kx, const void* x, long ldx, const void* w, const void* b, float alpha, int G,
                 int wlen, const void* gate, long ldg, const void* coef, float eps, void* out_f32, void* out, long ldo, void* h, long ldh, const void* scale,
                 cudaStream_t st) {
  if (M <= 0 || N <= 0) return 0;
  if (K % 8 || ldw % 8 || ((uintptr_t)W & 15) || M > 16 || kx > K || kx < 1 || pro < 0 || pro > 3) return cudaErrorInvalidValue;
  RowsArgs a{(const __nv_bfloat16*)W, ldw, N, K, M, pro, kx, x, ldx, (const float*)w, (const float*)b, alpha, G, wlen, (const float*)gate, ldg,
             (const float*)coef, eps, (float*)out_f32, (__nv_bfloat16*)out, ldo, (float*)h, ldh, (const float*)scale, 0};
  if (pro) {
    const int K32 = (K + 31) / 32 * 32;
    a.pitch = K32 * 2 + ((K32 * 2) % 128 == 0 ? 64 : 0);          // rows of a quad pair land in different halves of the banks
    if (M > 8 || (long)M * a.pitch > 200 * 1024) return cudaErrorInvalidValue;
    if ((pro == 1 && (!w || !b || h)) || (pro == 2 && (!w || G < 1 || kx % G || wlen < 1)) || (pro == 3 && !coef)) return cudaErrorInvalidValue;
  } else if (kx != K || ldx % 8 || ((uintptr_t)x & 15)) {
    return cudaErrorInvalidValue;
  }
  const int tiles = (N + 7) / 8;
  if (pro) {
    if (tiles <= 148 * 2) return launch_rows<8, true>(a, st);
    if (tiles <= 148 * 4) return launch_rows<4, true>(a, st);
    if (tiles <= 148 * 16) return launch_rows<2, true>(a, st);
    return launch_rows<1, true>(a, st);
  }
  if (tiles <= 148 * 4) return launch_rows<8, false>(a, st);
  if (tiles <= 148 * 8) return launch_rows<4, false>(a, st);
  if (tiles <= 148 * 16) return launch_rows<2, false>(a, st);
  return launch_rows<1, false>(a, st);
}

int ve_gemm_f32(const void* W, long ldw, const void* x, long ldx, void* out, long ldo, int T, int N, int K, cudaStream_t st) {
  if (T <= 0 || N <= 0) return 0;
  launch_pdl(gemm_f32_kernel, dim3((N + 63) / 64, (T + 63) / 64), dim3(256), 0, st, (const float*)W, ldw, (const float*)x, ldx, (float*)out, ldo, T, N, K);
  VE_CHECK_LAUNCH();
}

}  // extern "C"
