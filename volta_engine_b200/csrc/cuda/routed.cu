// Routed feed-forwards (mixture of experts) of decoders with an fp32 residual, weights in bf16 (or fp32 for the all-32-bit form):
//   route_rows   scores = softmax over all experts or the sigmoid of every logit, in fp32; experts come in equal groups of neighbours, only the best groups stay open (a
//                group's score: its best member, or the sum of its two best); the best open experts with their scores as weights
//                (optionally renormalised, times a factor); ties go to the lower index
//   routed_up    a few rows: routing, then gate and up rows of the chosen experts and the clamped gated unit (optionally of the input times the
//                weight: the weight then multiplies both products in front of the unit)
//   routed_down  a few rows: sum over a row's experts of weight * W_down a (or, behind weighted inputs, of W_down a), stored or added to the residual
// Prompt rows sort their routes by expert (moe.cu) and run the grouped tensor-core GEMM. Expert weights: gate_up [E][2 ff][ldg] (gate rows,
// then up rows), down [E][N][ldd]; row pitches are multiples of 16 bytes, pad columns are zero. No fast-math in this file.
#include "rowmath.cuh"
#include <float.h>

namespace ve {

struct Router {
  int E, top, groups, keep;
  int best2;                     // a group's score is the sum of its two best members
  int renorm; float factor;
  int sigmoid;                   // of every logit by itself, instead of the softmax
};
constexpr int kMaxExperts = 1024, kMaxTop = 32, kRoutedRows = 8;

VE_DEVINL int warp_argmax(float v, int i, float* best = nullptr) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float w = __shfl_xor_sync(0xffffffffu, v, o);
    const int k = __shfl_xor_sync(0xffffffffu, i, o);
    if (w > v || (w == v && k < i)) {
      v = w;
      i = k;
    }
  }
  if (best) *best = v;
  return i;
}

// One warp, one row. sc: E floats of scratch in shared memory, with groups > 1 `groups` more behind them: what experts and groups are ranked by
// (the softmax, or the logit: sigmoids near one cannot be told apart). A closed or taken expert's and a taken group's rank is -infinity.
VE_DEVINL void route_warp(const float* __restrict__ z, const Router& r, float* sc, int* ids, float* w) {
  const int lane = threadIdx.x & 31;
  const float NONE = __int_as_float(0xff800000);
  auto score = [&](float v) { return r.sigmoid ? sigmoid_of(v) : v; };
  float m = -FLT_MAX;
  for (int e = lane; e < r.E; e += 32) {
    float l = z[e];
    l = l != l ? -FLT_MAX : fminf(fmaxf(l, -FLT_MAX), FLT_MAX);        // a row of NaN must still give experts in range
    sc[e] = l;
    m = fmaxf(m, l);
  }
  if (!r.sigmoid) {
    m = warp_max(m);
    float s = 0.f;
    for (int e = lane; e < r.E; e += 32) {
      const float v = expf(sc[e] - m);
      sc[e] = v;
      s += v;
    }
    s = warp_sum(s);
    for (int e = lane; e < r.E; e += 32) sc[e] /= s;
  }
  __syncwarp();
  if (r.keep < r.groups) {
    float* gs = sc + r.E;
    const int per = r.E / r.groups;
    for (int g = lane; g < r.groups; g += 32) {
      float b1 = NONE, b2 = NONE;
      for (int e = g * per; e < (g + 1) * per; ++e) {
        const float v = sc[e];
        if (v > b1) {
          b2 = b1;
          b1 = v;
        } else if (v > b2) b2 = v;
      }
      gs[g] = r.best2 ? score(b1) + (per > 1 ? score(b2) : 0.f) : b1;
    }
    __syncwarp();
    for (int k = 0; k < r.keep; ++k) {
      float v = NONE;
      int i = 0x7fffffff;
      for (int g = lane; g < r.groups; g += 32)
        if (gs[g] > v) {
          v = gs[g];
          i = g;
        }
      i = warp_argmax(v, i);
      if (lane == 0) gs[i] = NONE;
      __syncwarp();
    }
    for (int e = lane; e < r.E; e += 32)
      if (gs[e / per] != NONE) sc[e] = NONE;
    __syncwarp();
  }
  float sum = 0.f;
  for (int k = 0; k < r.top; ++k) {
    float v = NONE;
    int i = 0x7fffffff;
    for (int e = lane; e < r.E; e += 32)
      if (sc[e] > v) {
        v = sc[e];
        i = e;
      }
    i = warp_argmax(v, i, &v);
    v = score(v);
    sum += v;
    if (lane == 0) {
      ids[k] = i;
      w[k] = v;
      sc[i] = NONE;
    }
    __syncwarp();
  }
  const float f = r.renorm ? r.factor / sum : r.factor;
  for (int k = lane; k < r.top; k += 32) w[k] *= f;
  __syncwarp();
}

// grid (rows / 8), a warp per row.
__global__ void __launch_bounds__(256) route_rows_kernel(const float* __restrict__ z, long ldz, int rows, const Router r, int* __restrict__ ids,
                                                         float* __restrict__ weights) {
  extern __shared__ float rsm[];            // [8][E + groups]
  __shared__ int s_id[8][kMaxTop];
  __shared__ float s_w[8][kMaxTop];
  grid_dep_wait();
  grid_dep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long row = blockIdx.x * 8l + warp;
  if (row >= rows) return;
  route_warp(z + row * ldz, r, rsm + warp * (r.E + r.groups), s_id[warp], s_w[warp]);
  if (lane < r.top) {
    ids[row * r.top + lane] = s_id[warp][lane];
    weights[row * r.top + lane] = s_w[warp][lane];
  }
}

// 16 bytes of a row in fp32
VE_DEVINL void load16(const __nv_bfloat16* p, float* o) {
  const uint4 t = *reinterpret_cast<const uint4*>(p);
  const uint32_t u[4] = {t.x, t.y, t.z, t.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    o[2 * j] = __uint_as_float(u[j] << 16);
    o[2 * j + 1] = __uint_as_float(u[j] & 0xffff0000u);
  }
}
VE_DEVINL void load16(const float* p, float* o) {
  const float4 t = *reinterpret_cast<const float4*>(p);
  o[0] = t.x; o[1] = t.y; o[2] = t.z; o[3] = t.w;
}
VE_DEVINL void dot16(const uint4 w, const __nv_bfloat16* x, float& acc) {
  float v[8];
  load16(x, v);
  const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    acc = fmaf(__uint_as_float(u[j] << 16), v[2 * j], acc);
    acc = fmaf(__uint_as_float(u[j] & 0xffff0000u), v[2 * j + 1], acc);
  }
}
VE_DEVINL void dot16(const uint4 w, const float* x, float& acc) {
  const float4 v = *reinterpret_cast<const float4*>(x);
  acc = fmaf(__uint_as_float(w.x), v.x, acc);
  acc = fmaf(__uint_as_float(w.y), v.y, acc);
  acc = fmaf(__uint_as_float(w.z), v.z, acc);
  acc = fmaf(__uint_as_float(w.w), v.w, acc);
}

struct RoutedUp {
  const float* z; long ldz;                // router logits
  Router r;
  int rows, R, K, ff;                      // R rows per group (grid.y)
  long ldx, ldw, lda;
  Glu unit;
  int* ids; float* weights;                // written by the first CTA of a group
  int wx;                                  // the weight multiplies what the expert reads
};

// grid (CTAs, row groups), 256 threads. X: rows as they are given (rounded to T). A warp makes one column of a route: gate and up row, lanes
// share K.
template <typename X, typename T>
__global__ void __launch_bounds__(256, 3) routed_up_kernel(const RoutedUp a, const X* __restrict__ x, const T* __restrict__ W, T* __restrict__ out) {
  constexpr int V = 16 / sizeof(T), U = 4;
  extern __shared__ __align__(16) uint8_t usm[];
  __shared__ int s_id[kRoutedRows][kMaxTop];
  __shared__ float s_w[kRoutedRows][kMaxTop];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, Kp = (a.K + V - 1) / V * V;
  T* xs = reinterpret_cast<T*>(usm);                             // [R][Kp]
  float* scratch = reinterpret_cast<float*>(xs + (size_t)a.R * Kp);
  const int row0 = blockIdx.y * a.R, n = min(a.R, a.rows - row0), top = a.r.top;
  grid_dep_wait();
  grid_dep_launch();
  if (warp < n) route_warp(a.z + (long)(row0 + warp) * a.ldz, a.r, scratch + warp * (a.r.E + a.r.groups), s_id[warp], s_w[warp]);
  for (int m = 0; m < n; ++m)
    for (int i = tid; i < Kp; i += 256) xs[(size_t)m * Kp + i] = from_f<T>(i < a.K ? to_f(x[(row0 + m) * a.ldx + i]) : 0.f);
  __syncthreads();
  if (blockIdx.x == 0)
    for (int i = tid; i < n * top; i += 256) {
      a.ids[(long)row0 * top + i] = s_id[i / top][i % top];
      a.weights[(long)row0 * top + i] = s_w[i / top][i % top];
    }
  const int chunks = (a.ff + 7) / 8, items = n * top * chunks;
  for (int it = blockIdx.x; it < items; it += gridDim.x) {
    const int route = it / chunks, o = (it - route * chunks) * 8 + warp, m = route / top;
    if (o >= a.ff) continue;
    const T* wg = W + ((long)s_id[m][route - m * top] * 2 * a.ff + o) * a.ldw;
    const T* wu = wg + (long)a.ff * a.ldw;
    const T* xr = xs + (size_t)m * Kp;
    float g = 0.f, u = 0.f;
    for (int k0 = lane * V; k0 < Kp; k0 += 32 * V * U) {
      uint4 p[U], q[U];
#pragma unroll
      for (int j = 0; j < U; ++j) {
        const int k = k0 + j * 32 * V;
        p[j] = k < Kp ? __ldcs(reinterpret_cast<const uint4*>(wg + k)) : make_uint4(0, 0, 0, 0);
        q[j] = k < Kp ? __ldcs(reinterpret_cast<const uint4*>(wu + k)) : make_uint4(0, 0, 0, 0);
      }
#pragma unroll
      for (int j = 0; j < U; ++j) {
        const int k = k0 + j * 32 * V;
        if (k < Kp) {
          dot16(p[j], xr + k, g);
          dot16(q[j], xr + k, u);
        }
      }
    }
    g = warp_sum(g);
    u = warp_sum(u);
    if (lane == 0) {
      const float f = a.wx ? s_w[m][route - m * top] : 1.f;
      out[((long)row0 * top + route) * a.lda + o] = from_f<T>(clamped_glu_of(g * f, u * f, a.unit));
    }
  }
}

struct RoutedDown {
  const int* ids; const float* weights;    // weights null: all one
  int top, N, ff;
  long lda, ldw, ldo;
  int add;                                 // out (fp32) is added to
};

// grid (CTAs, rows), 256 threads, a warp per output column. STAGED: activations in dynamic shared memory [top][ff rounded up to 16 bytes] of
// T; else they are read where they are (rows of whole 16-byte pieces).
template <bool STAGED, typename T, typename O>
__global__ void __launch_bounds__(256) routed_down_kernel(const RoutedDown a, const T* __restrict__ act, const T* __restrict__ W, O* __restrict__ out) {
  constexpr int V = 16 / sizeof(T), U = 4;
  extern __shared__ __align__(16) uint8_t dsm[];
  __shared__ int s_id[kMaxTop];
  __shared__ float s_w[kMaxTop];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, F = (a.ff + V - 1) / V * V;
  const long row = blockIdx.y;
  const T* as = STAGED ? reinterpret_cast<const T*>(dsm) : act + row * a.top * a.lda;
  const long pitch = STAGED ? F : a.lda;
  grid_dep_wait();
  grid_dep_launch();
  if (tid < a.top) {
    s_id[tid] = a.ids[row * a.top + tid];
    s_w[tid] = a.weights ? a.weights[row * a.top + tid] : 1.f;
  }
  if (STAGED)
    for (int i = tid; i < a.top * F; i += 256) {
      const int k = i / F, f = i - k * F;
      reinterpret_cast<T*>(dsm)[i] = f < a.ff ? act[(row * a.top + k) * a.lda + f] : from_f<T>(0.f);
    }
  __syncthreads();
  for (int n = blockIdx.x * 8 + warp; n < a.N; n += gridDim.x * 8) {
    float acc = 0.f;
    for (int k0 = 0; k0 < a.top; k0 += U) {
      float d[U] = {0.f, 0.f, 0.f, 0.f};
      for (int f = lane * V; f < F; f += 32 * V) {
        uint4 p[U];
#pragma unroll
        for (int j = 0; j < U; ++j)
          p[j] = k0 + j < a.top ? __ldcs(reinterpret_cast<const uint4*>(W + ((long)s_id[k0 + j] * a.N + n) * a.ldw + f)) : make_uint4(0, 0, 0, 0);
#pragma unroll
        for (int j = 0; j < U; ++j)
          if (k0 + j < a.top) dot16(p[j], as + (k0 + j) * pitch + f, d[j]);
      }
#pragma unroll
      for (int j = 0; j < U; ++j)
        if (k0 + j < a.top) acc = fmaf(s_w[k0 + j], d[j], acc);
    }
    acc = warp_sum(acc);
    if (lane == 0) out[row * a.ldo + n] = from_f<O>(a.add ? acc + to_f(out[row * a.ldo + n]) : acc);
  }
}

template <typename F>
static int routed_smem(F kernel, size_t smem, size_t& have) {
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  if (smem <= have || smem <= 40 * 1024) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e == cudaSuccess) have = smem;
  return (int)e;
}
template <typename X, typename T>
static int launch_routed_up(RoutedUp a, const void* x, const void* W, void* out, cudaStream_t st) {
  constexpr int V = 16 / sizeof(T);
  const size_t row = (size_t)((a.K + V - 1) / V * V) * sizeof(T) + (size_t)(a.r.E + a.r.groups) * 4;
  a.R = kRoutedRows;
  while (a.R > 1 && (a.R * row > 64 * 1024 || a.R / 2 >= a.rows)) a.R /= 2;
  static size_t have = 0;
  const int rc = routed_smem(routed_up_kernel<X, T>, a.R * row, have);
  if (rc) return rc;
  const int groups = (a.rows + a.R - 1) / a.R;
  const long items = (long)a.R * a.r.top * ((a.ff + 7) / 8), room = groups >= 444 ? 1 : 444 / groups, per = (items + room - 1) / room;
  launch_pdl(routed_up_kernel<X, T>, dim3((unsigned)((items + per - 1) / per), groups), dim3(256), a.R * row, st, a, (const X*)x, (const T*)W, (T*)out);
  return (int)cudaGetLastError();
}
template <typename T, typename O>
static int launch_routed_down(const RoutedDown& a, const void* act, const void* W, void* out, int rows, cudaStream_t st) {
  constexpr int V = 16 / sizeof(T);
  const size_t smem = (size_t)a.top * ((a.ff + V - 1) / V * V) * sizeof(T);
  const int chunks = (a.N + 7) / 8, room = rows >= 592 ? 1 : 592 / rows, per = (chunks + room - 1) / room;
  const dim3 grid((chunks + per - 1) / per, rows);
  if (smem > 96 * 1024 && a.ff % V == 0 && a.lda % V == 0 && !((uintptr_t)act & 15)) {
    launch_pdl(routed_down_kernel<false, T, O>, grid, dim3(256), 0, st, a, (const T*)act, (const T*)W, (O*)out);
    return (int)cudaGetLastError();
  }
  static size_t have = 0;
  const int rc = routed_smem(routed_down_kernel<true, T, O>, smem, have);
  if (rc) return rc;
  launch_pdl(routed_down_kernel<true, T, O>, grid, dim3(256), smem, st, a, (const T*)act, (const T*)W, (O*)out);
  return (int)cudaGetLastError();
}

}  // namespace ve

using namespace ve;

#define VE_ROUTER int E, int top, int groups, int keep, int best2, int renorm, float factor, int sigmoid
#define VE_RMAKE Router{E, top, groups, keep, best2, renorm, factor, sigmoid}
static bool router_ok(const Router& r) {
  return r.E > 0 && r.E <= kMaxExperts && r.top > 0 && r.top <= kMaxTop && r.groups > 0 && r.E % r.groups == 0 && r.keep > 0 && r.keep <= r.groups &&
         r.top <= r.keep * (r.E / r.groups);
}

extern "C" {

int ve_route_rows(VE_ROUTER, const void* z, long ldz, void* ids, void* weights, int rows, cudaStream_t st) {
  if (rows <= 0) return 0;
  const Router r = VE_RMAKE;
  if (!router_ok(r)) return cudaErrorInvalidValue;
  static size_t have = 0;
  const size_t smem = (size_t)8 * (E + groups) * 4;
  const int rc = routed_smem(route_rows_kernel, smem, have);
  if (rc) return rc;
  launch_pdl(route_rows_kernel, dim3((rows + 7) / 8), dim3(256), smem, st, (const float*)z, ldz, rows, r, (int*)ids, (float*)weights);
  VE_CHECK_LAUNCH();
}

// x [rows][K] fp32 when x32, else of the weights' type; f32: weights and output fp32 (else bf16). out [rows top][lda]; ids, weights
// [rows][top] are written. wx: the weights multiply the inputs.
int ve_routed_up(VE_ROUTER, const void* z, long ldz, const void* x, long ldx, int x32, const void* W, long ldw, void* out, long lda, void* ids, void* weights,
                 int rows, int K, int ff, float alpha, float limit, float shift, int wx, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const Router r = VE_RMAKE;
  if (!router_ok(r) || K < 1 || ff < 1 || (ldw * (f32 ? 4 : 2)) % 16 || ((uintptr_t)W & 15) || ldw < K) return cudaErrorInvalidValue;
  const RoutedUp a{(const float*)z, ldz, r, rows, 0, K, ff, ldx, ldw, lda, Glu{alpha, limit, shift}, (int*)ids, (float*)weights, wx};
  if (f32) return launch_routed_up<float, float>(a, x, W, out, st);
  if (x32) return launch_routed_up<float, __nv_bfloat16>(a, x, W, out, st);
  return launch_routed_up<__nv_bfloat16, __nv_bfloat16>(a, x, W, out, st);
}

// act [rows top][lda] of the weights' type; out [rows][ldo] fp32 when o32 or f32, else bf16; add: out fp32 is added to. weights null: all one.
int ve_routed_down(const void* act, long lda, const void* W, long ldw, const void* ids, const void* weights, int top, void* out, long ldo, int o32, int rows,
                   int N, int ff, int add, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (top < 1 || top > kMaxTop || N < 1 || ff < 1 || (ldw * (f32 ? 4 : 2)) % 16 || ((uintptr_t)W & 15) || ldw < ff || (add && !o32 && !f32)) return cudaErrorInvalidValue;
  const RoutedDown a{(const int*)ids, (const float*)weights, top, N, ff, lda, ldw, ldo, add};
  if (f32) return launch_routed_down<float, float>(a, act, W, out, rows, st);
  if (o32) return launch_routed_down<__nv_bfloat16, float>(a, act, W, out, rows, st);
  return launch_routed_down<__nv_bfloat16, __nv_bfloat16>(a, act, W, out, rows, st);
}

}  // extern "C"
