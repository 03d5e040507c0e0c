// Row operators of decoders whose residual stream is fp32. Storage of activations is a template parameter (bf16, or fp32
// for the all-32-bit form of a model); every operator computes in fp32. This file is compiled without fast-math: norms,
// gates and angles follow the 32-bit definitions to rounding.
//   embed_rows   out[r] = table[ids[r]] widened to fp32
//   dyt_rows     h += scale * part (optional, element-wise scale), out = tanh(alpha h) w + b        ("Dynamic Tanh" norm)
//   group_rms    out = x / rms(x over groups of G columns) * w [* sigmoid(gate)]; w repeats with its own length
//   polynorm     out = c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3, N = division by the row's root mean square
//   scale_add    h += scale * part
#include "rowmath.cuh"

namespace ve {

template <typename T>
__global__ void embed_rows_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out, int H, int vocab) {
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  int id = ids[row];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  for (int i = threadIdx.x; i < H; i += blockDim.x) out[row * H + i] = to_f(table[(long)id * H + i]);
}

template <typename T>
__global__ void dyt_rows_kernel(float* __restrict__ h, const T* __restrict__ part, long ldp, const float* __restrict__ scale,
                                const float* __restrict__ w, const float* __restrict__ b, float alpha, T* __restrict__ out,
                                long ldo, int H) {
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  float* hr = h + row * H;
  const int per = (H + gridDim.y - 1) / gridDim.y, i0 = blockIdx.y * per, i1 = min(H, i0 + per);
  for (int i = i0 + threadIdx.x; i < i1; i += blockDim.x) {
    float v = hr[i];
    if (part) {
      v = fmaf(to_f(part[row * ldp + i]), scale ? scale[i] : 1.f, v);
      hr[i] = v;
    }
    if (out) out[row * ldo + i] = from_f<T>(dyt_of(v, alpha, w[i], b[i]));
  }
}

// The same on four columns per thread (H, the pitches and all bases multiples of four elements).
template <typename T>
__global__ void dyt_rows4_kernel(float* __restrict__ h, const T* __restrict__ part, long ldp, const float* __restrict__ scale,
                                 const float* __restrict__ w, const float* __restrict__ b, float alpha, T* __restrict__ out,
                                 long ldo, int H, long total4) {
  grid_dep_wait();
  grid_dep_launch();
  const int h4 = H >> 2;
  for (long q = blockIdx.x * (long)blockDim.x + threadIdx.x; q < total4; q += (long)gridDim.x * blockDim.x) {
    const long row = q / h4;
    const int i = (int)(q - row * h4) * 4;
    float4 v = *reinterpret_cast<const float4*>(h + row * H + i);
    if (part) {
      const float4 p = load4(part + row * ldp + i);
      const float4 s = scale ? *reinterpret_cast<const float4*>(scale + i) : make_float4(1.f, 1.f, 1.f, 1.f);
      v.x = fmaf(p.x, s.x, v.x);
      v.y = fmaf(p.y, s.y, v.y);
      v.z = fmaf(p.z, s.z, v.z);
      v.w = fmaf(p.w, s.w, v.w);
      *reinterpret_cast<float4*>(h + row * H + i) = v;
    }
    if (out) {
      const float4 wv = *reinterpret_cast<const float4*>(w + i), bv = *reinterpret_cast<const float4*>(b + i);
      store4(out + row * ldo + i, make_float4(dyt_of(v.x, alpha, wv.x, bv.x), dyt_of(v.y, alpha, wv.y, bv.y),
                                              dyt_of(v.z, alpha, wv.z, bv.z), dyt_of(v.w, alpha, wv.w, bv.w)));
    }
  }
}

// grid (rows, groups); x fp32 or T
template <typename X, typename T>
__global__ void group_rms_kernel(const X* __restrict__ x, long ldx, const float* __restrict__ w, int wlen, const X* __restrict__ gate,
                                 long ldg, T* __restrict__ out, long ldo, int G, float eps) {
  __shared__ float red[33];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  const int c0 = blockIdx.y * G;
  float ss = 0.f;
  for (int i = threadIdx.x; i < G; i += blockDim.x) {
    const float v = to_f(x[row * ldx + c0 + i]);
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)G + eps);
  for (int i = threadIdx.x; i < G; i += blockDim.x) {
    const int c = c0 + i;
    float v = to_f(x[row * ldx + c]) * inv * w[c % wlen];
    if (gate) v *= sigmoid_of(to_f(gate[row * ldg + c]));
    out[row * ldo + c] = from_f<T>(v);
  }
}

template <typename X, typename T>
__global__ void __launch_bounds__(256) polynorm_kernel(const X* __restrict__ z, long ldz, const float* __restrict__ coef, T* __restrict__ out, long ldo,
                                                       int F, float eps) {
  __shared__ float red[33];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  for (int i = threadIdx.x; i < F; i += blockDim.x) poly_sums(to_f(z[row * ldz + i]), s1, s2, s3);
  s1 = block_sum(s1, red);
  s2 = block_sum(s2, red);
  s3 = block_sum(s3, red);
  const PolyScale ps = poly_scale(s1, s2, s3, F, eps, coef);
  for (int i = threadIdx.x; i < F; i += blockDim.x) out[row * ldo + i] = from_f<T>(poly_of(to_f(z[row * ldz + i]), ps));
}

// One pass over global memory: every thread keeps its 8-wide slices of the row in registers (F <= 256 * 8 * N8).
template <int N8>
__global__ void __launch_bounds__(256) polynorm8_kernel(const __nv_bfloat16* __restrict__ z, long ldz, const float* __restrict__ coef,
                                                        __nv_bfloat16* __restrict__ out, long ldo, int F, float eps) {
  __shared__ float red[33];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  bf16x8 v[N8];
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
  for (int j = 0; j < N8; ++j) {
    const int i = (j * 256 + threadIdx.x) * 8;
    if (i < F) {
      v[j] = *reinterpret_cast<const bf16x8*>(z + row * ldz + i);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(v[j].v[e]);
        poly_sums(f.x, s1, s2, s3);
        poly_sums(f.y, s1, s2, s3);
      }
    }
  }
  s1 = block_sum(s1, red);
  s2 = block_sum(s2, red);
  s3 = block_sum(s3, red);
  const PolyScale ps = poly_scale(s1, s2, s3, F, eps, coef);
#pragma unroll
  for (int j = 0; j < N8; ++j) {
    const int i = (j * 256 + threadIdx.x) * 8;
    if (i < F) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(v[j].v[e]);
        v[j].v[e] = __floats2bfloat162_rn(poly_of(f.x, ps), poly_of(f.y, ps));
      }
      *reinterpret_cast<bf16x8*>(out + row * ldo + i) = v[j];
    }
  }
}

static inline int row_threads(int n) { return n >= 1024 ? 256 : n >= 256 ? 128 : ((n + 31) / 32 * 32 < 32 ? 32 : (n + 31) / 32 * 32); }

}  // namespace ve

using namespace ve;

extern "C" {

// f32: 1 = activations and tables fp32, 0 = bf16.
int ve_embed_rows(const void* ids, const void* table, void* out, int rows, int H, int vocab, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (f32) launch_pdl(embed_rows_kernel<float>, dim3(rows), dim3(row_threads(H)), 0, st, (const int*)ids, (const float*)table, (float*)out, H, vocab);
  else launch_pdl(embed_rows_kernel<__nv_bfloat16>, dim3(rows), dim3(row_threads(H)), 0, st, (const int*)ids, (const __nv_bfloat16*)table, (float*)out, H, vocab);
  VE_CHECK_LAUNCH();
}

// part, scale and out may be null. h [rows, H] contiguous fp32.
int ve_dyt_rows(void* h, const void* part, long ldp, const void* scale, const void* w, const void* b, float alpha, void* out, long ldo,
                int rows, int H, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const bool vec = !f32 && H % 4 == 0 && (!part || ldp % 4 == 0) && (!out || ldo % 4 == 0) && !((uintptr_t)h & 15) && !((uintptr_t)part & 7) &&
                   !((uintptr_t)scale & 15) && !((uintptr_t)w & 15) && !((uintptr_t)b & 15) && !((uintptr_t)out & 7);
  if (vec) {
    const long total4 = (long)rows * (H / 4);
    const long blocks = (total4 + 255) / 256;
    launch_pdl(dyt_rows4_kernel<__nv_bfloat16>, dim3((unsigned)(blocks < 148 * 8 ? blocks : 148 * 8)), dim3(256), 0, st, (float*)h, (const __nv_bfloat16*)part,
               ldp, (const float*)scale, (const float*)w, (const float*)b, alpha, (__nv_bfloat16*)out, ldo, H, total4);
    VE_CHECK_LAUNCH();
  }
  const dim3 grid(rows, rows >= 148 ? 1 : (H + 1023) / 1024);
  if (f32) launch_pdl(dyt_rows_kernel<float>, grid, dim3(row_threads(H)), 0, st, (float*)h, (const float*)part, ldp, (const float*)scale,
                      (const float*)w, (const float*)b, alpha, (float*)out, ldo, H);
  else launch_pdl(dyt_rows_kernel<__nv_bfloat16>, grid, dim3(row_threads(H)), 0, st, (float*)h, (const __nv_bfloat16*)part, ldp,
                  (const float*)scale, (const float*)w, (const float*)b, alpha, (__nv_bfloat16*)out, ldo, H);
  VE_CHECK_LAUNCH();
}

// x (and gate) fp32 when x32, else of the activation type; cols = groups * G.
int ve_group_rms(const void* x, long ldx, int x32, const void* w, int wlen, const void* gate, long ldg, void* out, long ldo, int rows, int cols,
                 int G, float eps, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (G <= 0 || cols % G || wlen <= 0) return cudaErrorInvalidValue;
  const dim3 grid(rows, cols / G), block(row_threads(G));
#define VE_GR(X, T) launch_pdl(group_rms_kernel<X, T>, grid, block, 0, st, (const X*)x, ldx, (const float*)w, wlen, (const X*)gate, ldg, (T*)out, ldo, G, eps)
  if (f32) VE_GR(float, float);
  else if (x32) VE_GR(float, __nv_bfloat16);
  else VE_GR(__nv_bfloat16, __nv_bfloat16);
#undef VE_GR
  VE_CHECK_LAUNCH();
}

int ve_polynorm(const void* z, long ldz, int x32, const void* coef, void* out, long ldo, int rows, int F, float eps, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const bool vec = !f32 && !x32 && F % 8 == 0 && ldz % 8 == 0 && ldo % 8 == 0 && !((uintptr_t)z & 15) && !((uintptr_t)out & 15);
#define VE_PN8(N8) launch_pdl(polynorm8_kernel<N8>, dim3(rows), dim3(256), 0, st, (const __nv_bfloat16*)z, ldz, (const float*)coef, (__nv_bfloat16*)out, ldo, F, eps)
  if (vec && F <= 2048) VE_PN8(1);
  else if (vec && F <= 8192) VE_PN8(4);
  else if (vec && F <= 16384) VE_PN8(8);
  else {
    const dim3 block(row_threads(F));
#define VE_PN(X, T) launch_pdl(polynorm_kernel<X, T>, dim3(rows), block, 0, st, (const X*)z, ldz, (const float*)coef, (T*)out, ldo, F, eps)
    if (f32) VE_PN(float, float);
    else if (x32) VE_PN(float, __nv_bfloat16);
    else VE_PN(__nv_bfloat16, __nv_bfloat16);
#undef VE_PN
  }
#undef VE_PN8
  VE_CHECK_LAUNCH();
}

}  // extern "C"
