// Row operators of decoders whose residual stream is fp32. Storage of activations is a template parameter (bf16, or fp32
// for the all-32-bit form of a model); every operator computes in fp32. This file is compiled without fast-math: norms,
// gates and angles follow the 32-bit definitions to rounding.
//   embed_rows   out[r] = table[ids[r]] widened to fp32, times a scale [+ sinusoidal position vector], once per residual stream
//   dyt_rows     h += scale * part (optional, element-wise scale), out = tanh(alpha h) w + b        ("Dynamic Tanh" norm)
//   stream_norm  residual streams rewritten from the old ones and a sublayer's result (optional), then the layer norm (no shift) of
//                their weighted sum
//   group_rms    out = x / rms(x over groups of G columns) * w [* sigmoid(gate) or silu(gate)]; w repeats with its own length
//   residual_norm  h += a sublayer's result (or the weighted sum of a token's routed results) or its RMS norm, out = h or its RMS norm
//   clamped_glu  out = gated unit of [gate | up] rows (optionally times a weight per row) with both halves clamped
//   soft_cap     x = cap tanh(x / cap)
//   polynorm     out = c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3, N = division by the row's root mean square
//   scale_add    h += scale * part
#include "rowmath.cuh"

namespace ve {

// freq (optional, double): turns by half circles per position and column pair; column 2i gets the sine, 2i + 1 the cosine.
template <typename T>
__global__ void embed_rows_kernel(const int* __restrict__ ids, const T* __restrict__ table, const int* __restrict__ pos, const double* __restrict__ freq,
                                  float* __restrict__ out, int H, int vocab, int S, float scale) {
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  int id = ids[row];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* src = table + (long)id * H;
  float* dst = out + row * S * H;
  if (!freq) {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float v = to_f(src[i]) * scale;
      for (int s = 0; s < S; ++s) dst[(long)s * H + i] = v;
    }
    return;
  }
  const double p = (double)pos[row];
  for (int i = threadIdx.x * 2; i < H; i += blockDim.x * 2) {
    const double t = p * freq[i >> 1];
    float sn, cs;
    sincospif((float)(t - 2.0 * rint(0.5 * t)), &sn, &cs);
    const float v0 = fmaf(to_f(src[i]), scale, sn), v1 = i + 1 < H ? fmaf(to_f(src[i + 1]), scale, cs) : 0.f;
    for (int s = 0; s < S; ++s) {
      dst[(long)s * H + i] = v0;
      if (i + 1 < H) dst[(long)s * H + i + 1] = v1;
    }
  }
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

VE_DEVINL float gate_of(float z, int silu) { return silu ? silu_of(z) : sigmoid_of(z); }

// grid (rows, groups); x fp32 or T
template <typename X, typename T>
__global__ void group_rms_kernel(const X* __restrict__ x, long ldx, const float* __restrict__ w, int wlen, const X* __restrict__ gate,
                                 long ldg, int silu, T* __restrict__ out, long ldo, int G, float eps) {
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
    if (gate) v *= gate_of(to_f(gate[row * ldg + c]), silu);
    out[row * ldo + c] = from_f<T>(v);
  }
}

// Narrow groups (G <= 128 N4): one warp per group, the group in registers, four columns per lane and step (G, wlen, pitches and
// bases multiples of four elements). groups = all groups of all rows.
template <int N4, typename X, typename T>
__global__ void __launch_bounds__(256) group_rms4_kernel(const X* __restrict__ x, long ldx, const float* __restrict__ w, int wlen, const X* __restrict__ gate,
                                                         long ldg, int silu, T* __restrict__ out, long ldo, int G, int per_row, long groups, float eps) {
  grid_dep_wait();
  grid_dep_launch();
  const int lane = threadIdx.x & 31;
  for (long q = blockIdx.x * 8l + (threadIdx.x >> 5); q < groups; q += gridDim.x * 8l) {
    const long row = q / per_row;
    const int c0 = (int)(q - row * per_row) * G;
    float4 v[N4], z[N4];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < N4; ++j) {
      const int i = (j * 32 + lane) * 4;
      v[j] = i < G ? load4(x + row * ldx + c0 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      if (gate && i < G) z[j] = load4(gate + row * ldg + c0 + i);
      ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)G + eps);
#pragma unroll
    for (int j = 0; j < N4; ++j) {
      const int i = (j * 32 + lane) * 4;
      if (i >= G) continue;
      const float4 wv = *reinterpret_cast<const float4*>(w + (c0 + i) % wlen);
      float4 o = make_float4(v[j].x * inv * wv.x, v[j].y * inv * wv.y, v[j].z * inv * wv.z, v[j].w * inv * wv.w);
      if (gate) {
        o.x *= gate_of(z[j].x, silu);
        o.y *= gate_of(z[j].y, silu);
        o.z *= gate_of(z[j].z, silu);
        o.w *= gate_of(z[j].w, silu);
      }
      store4(out + row * ldo + c0 + i, o);
    }
  }
}

// h [rows][S][H]. One CTA per row.
template <typename T>
__global__ void __launch_bounds__(256) stream_norm_kernel(float* __restrict__ h, const T* __restrict__ part, long ldp, const float* __restrict__ mix,
                                                          const float* __restrict__ wout, const float* __restrict__ win, const float* __restrict__ w,
                                                          T* __restrict__ out, long ldo, int H, int S, float eps) {
  __shared__ float red[33];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  float* hr = h + row * S * H;
  auto read = [&](int i) {
    float u = 0.f;
    for (int s = 0; s < S; ++s) u = fmaf(win[s], hr[(long)s * H + i], u);
    return u;
  };
  float sum = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    if (part) {
      float x[kMaxStreams];
#pragma unroll
      for (int s = 0; s < kMaxStreams; ++s) x[s] = s < S ? hr[(long)s * H + i] : 0.f;
      streams_write(x, S, mix, wout, to_f(part[row * ldp + i]));
#pragma unroll
      for (int s = 0; s < kMaxStreams; ++s)
        if (s < S) hr[(long)s * H + i] = x[s];
    }
    if (out) sum += read(i);                              // (a thread reads what it wrote itself)
  }
  if (!out) return;
  const float mean = block_sum(sum, red) / (float)H;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float d = read(i) - mean;
    ss = fmaf(d, d, ss);
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)H + eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x) out[row * ldo + i] = from_f<T>((read(i) - mean) * inv * w[i]);
}

// The same on four columns per thread and step, the row in registers (H <= 1024 NV; H, pitches and bases multiples of four).
template <int S, int NV, typename T>
__global__ void __launch_bounds__(256) stream_norm4_kernel(float* __restrict__ h, const T* __restrict__ part, long ldp, const float* __restrict__ mix,
                                                           const float* __restrict__ wout, const float* __restrict__ win, const float* __restrict__ w,
                                                           T* __restrict__ out, long ldo, int H, float eps) {
  __shared__ float red[33];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  float* hr = h + row * S * H;
  float a[S][S], b[S], r[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    r[s] = win[s];
    b[s] = part ? wout[s] : 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) a[s][t] = part ? mix[s * S + t] : 0.f;
  }
  float4 u[NV];
  float sum = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (j * 256 + threadIdx.x) * 4;
    u[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < H) {
      float4 x[S];
#pragma unroll
      for (int s = 0; s < S; ++s) x[s] = *reinterpret_cast<const float4*>(hr + (long)s * H + i);
      if (part) {
        const float4 p = load4(part + row * ldp + i);
        float4 y[S];
#pragma unroll
        for (int t = 0; t < S; ++t) {
          y[t] = make_float4(b[t] * p.x, b[t] * p.y, b[t] * p.z, b[t] * p.w);
#pragma unroll
          for (int s = 0; s < S; ++s) {
            y[t].x = fmaf(a[s][t], x[s].x, y[t].x);
            y[t].y = fmaf(a[s][t], x[s].y, y[t].y);
            y[t].z = fmaf(a[s][t], x[s].z, y[t].z);
            y[t].w = fmaf(a[s][t], x[s].w, y[t].w);
          }
          *reinterpret_cast<float4*>(hr + (long)t * H + i) = y[t];
        }
#pragma unroll
        for (int s = 0; s < S; ++s) x[s] = y[s];
      }
#pragma unroll
      for (int s = 0; s < S; ++s) {
        u[j].x = fmaf(r[s], x[s].x, u[j].x);
        u[j].y = fmaf(r[s], x[s].y, u[j].y);
        u[j].z = fmaf(r[s], x[s].z, u[j].z);
        u[j].w = fmaf(r[s], x[s].w, u[j].w);
      }
      sum += (u[j].x + u[j].y) + (u[j].z + u[j].w);
    }
  }
  if (!out) return;
  const float mean = block_sum(sum, red) / (float)H;
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    if ((j * 256 + threadIdx.x) * 4 < H) {
      u[j].x -= mean;
      u[j].y -= mean;
      u[j].z -= mean;
      u[j].w -= mean;
      ss += (u[j].x * u[j].x + u[j].y * u[j].y) + (u[j].z * u[j].z + u[j].w * u[j].w);
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)H + eps);
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (j * 256 + threadIdx.x) * 4;
    if (i < H) {
      const float4 wv = *reinterpret_cast<const float4*>(w + i);
      store4(out + row * ldo + i, make_float4(u[j].x * inv * wv.x, u[j].y * inv * wv.y, u[j].z * inv * wv.z, u[j].w * inv * wv.w));
    }
  }
}

// One sublayer result per row: rows of `part`, or (top > 0) sum_k rw[row][k] part[inv ? inv[row top + k] : row top + k] (rw null: all one).
struct ResultRows {
  const int* inv; const float* rw; int top;
};
// h [rows][H]. One CTA per row. part null: no result; wa null: the result as it is, not normed; wo null: the residual itself; out null: only the
// residual.
template <typename T>
__global__ void __launch_bounds__(256) residual_norm_kernel(float* __restrict__ h, const T* __restrict__ part, long ldp, const ResultRows rr,
                                                            const float* __restrict__ wa, const float* __restrict__ wo, T* __restrict__ out, long ldo, int H,
                                                            float eps) {
  __shared__ float red[33];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  float* hr = h + row * H;
  auto result = [&](int i) {
    if (!rr.top) return to_f(part[row * ldp + i]);
    float v = 0.f;
    for (int k = 0; k < rr.top; ++k) {
      const long r = row * rr.top + k;
      v = fmaf(rr.rw ? rr.rw[r] : 1.f, to_f(part[(rr.inv ? rr.inv[r] : r) * ldp + i]), v);
    }
    return v;
  };
  float inv = 0.f, s = 0.f;
  if (wa) {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float v = result(i);
      s = fmaf(v, v, s);
    }
    inv = 1.f / sqrtf(block_sum(s, red) / (float)H + eps);
    s = 0.f;
  }
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float v = hr[i];
    if (part) {
      v = wa ? fmaf(result(i) * inv, wa[i], v) : v + result(i);
      hr[i] = v;
    }
    if (!out) continue;
    if (!wo) out[row * ldo + i] = from_f<T>(v);
    s = fmaf(v, v, s);
  }
  if (!out || !wo) return;
  inv = 1.f / sqrtf(block_sum(s, red) / (float)H + eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x) out[row * ldo + i] = from_f<T>(hr[i] * inv * wo[i]);      // (a thread reads what it wrote itself)
}

// The same on four columns per thread and step, the row in registers (H <= 1024 NV; H, pitches and bases multiples of four).
template <int NV, typename T>
__global__ void __launch_bounds__(256) residual_norm4_kernel(float* __restrict__ h, const T* __restrict__ part, long ldp, const ResultRows rr,
                                                             const float* __restrict__ wa, const float* __restrict__ wo, T* __restrict__ out, long ldo, int H,
                                                             float eps) {
  __shared__ float red[33];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  float* hr = h + row * H;
  float4 y[NV], x[NV];
  float s = 0.f;
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (j * 256 + threadIdx.x) * 4;
    x[j] = i < H ? load4(hr + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    y[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (part && !rr.top && i < H) y[j] = load4(part + row * ldp + i);
  }
  if (part) {
    for (int k = 0; k < rr.top; ++k) {
      const long r = row * rr.top + k;
      const T* pr = part + (rr.inv ? rr.inv[r] : r) * ldp;
      const float f = rr.rw ? rr.rw[r] : 1.f;
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const int i = (j * 256 + threadIdx.x) * 4;
        if (i < H) {
          const float4 v = load4(pr + i);
          y[j] = make_float4(fmaf(f, v.x, y[j].x), fmaf(f, v.y, y[j].y), fmaf(f, v.z, y[j].z), fmaf(f, v.w, y[j].w));
        }
      }
    }
    float inv = 1.f;
    if (wa) {
#pragma unroll
      for (int j = 0; j < NV; ++j) s += (y[j].x * y[j].x + y[j].y * y[j].y) + (y[j].z * y[j].z + y[j].w * y[j].w);
      inv = 1.f / sqrtf(block_sum(s, red) / (float)H + eps);
      s = 0.f;
    }
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = (j * 256 + threadIdx.x) * 4;
      if (i < H) {
        const float4 w = wa ? load4(wa + i) : make_float4(1.f, 1.f, 1.f, 1.f);
        x[j] = make_float4(fmaf(y[j].x * inv, w.x, x[j].x), fmaf(y[j].y * inv, w.y, x[j].y), fmaf(y[j].z * inv, w.z, x[j].z), fmaf(y[j].w * inv, w.w, x[j].w));
        store4(hr + i, x[j]);
      }
    }
  }
  if (!out) return;
  float inv = 1.f;
  if (wo) {
#pragma unroll
    for (int j = 0; j < NV; ++j) s += (x[j].x * x[j].x + x[j].y * x[j].y) + (x[j].z * x[j].z + x[j].w * x[j].w);
    inv = 1.f / sqrtf(block_sum(s, red) / (float)H + eps);
  }
#pragma unroll
  for (int j = 0; j < NV; ++j) {
    const int i = (j * 256 + threadIdx.x) * 4;
    if (i >= H) continue;
    if (wo) {
      const float4 w = load4(wo + i);
      x[j] = make_float4(x[j].x * inv * w.x, x[j].y * inv * w.y, x[j].z * inv * w.z, x[j].w * inv * w.w);
    }
    store4(out + row * ldo + i, x[j]);
  }
}

__global__ void __launch_bounds__(256) soft_cap_kernel(float* __restrict__ x, long n, float cap) {
  grid_dep_wait();
  grid_dep_launch();
  for (long i = blockIdx.x * 256l + threadIdx.x; i < n; i += gridDim.x * 256l) x[i] = soft_cap_of(x[i], cap);
}

// Factor of a row: w[index[row]] (w null: one).
struct RowBy {
  const float* w; const int* index;
  VE_DEVINL float of(long row) const { return w ? w[index[row]] : 1.f; }
};

// z [rows][2 F]: gates, then ups (blk 0), or blocks of [4 gates | 4 ups].
template <typename X, typename T>
__global__ void __launch_bounds__(256) clamped_glu_kernel(const X* __restrict__ z, long ldz, T* __restrict__ out, long ldo, long total, int F, int blk, const Glu u, const RowBy by) {
  grid_dep_wait();
  grid_dep_launch();
  for (long q = blockIdx.x * 256l + threadIdx.x; q < total; q += gridDim.x * 256l) {
    const long row = q / F;
    const int i = (int)(q - row * F), g = blk ? (i >> 2) * 8 + (i & 3) : i, up = blk ? g + 4 : F + i;
    const float f = by.of(row);
    out[row * ldo + i] = from_f<T>(clamped_glu_of(to_f(z[row * ldz + g]) * f, to_f(z[row * ldz + up]) * f, u));
  }
}
VE_DEVINL __nv_bfloat162 clamped_glu2(__nv_bfloat162 g, __nv_bfloat162 u, const Glu& c, float f) {
  const float2 a = __bfloat1622float2(g), b = __bfloat1622float2(u);
  return __floats2bfloat162_rn(clamped_glu_of(a.x * f, b.x * f, c), clamped_glu_of(a.y * f, b.y * f, c));
}
__global__ void __launch_bounds__(256) clamped_glu8_kernel(const __nv_bfloat16* __restrict__ z, long ldz, __nv_bfloat16* __restrict__ out, long ldo, long total8,
                                                           int F, int blk, const Glu u, const RowBy by) {
  grid_dep_wait();
  grid_dep_launch();
  const int f8 = F >> 3;
  for (long q = blockIdx.x * 256l + threadIdx.x; q < total8; q += gridDim.x * 256l) {
    const long row = q / f8;
    const int i = (int)(q - row * f8) * 8;
    const __nv_bfloat16* zr = z + row * ldz;
    const bf16x8 a = *reinterpret_cast<const bf16x8*>(zr + (blk ? 2 * i : i)), b = *reinterpret_cast<const bf16x8*>(zr + (blk ? 2 * i + 8 : F + i));
    const float f = by.of(row);
    bf16x8 o;
    if (blk) {
      o.v[0] = clamped_glu2(a.v[0], a.v[2], u, f);
      o.v[1] = clamped_glu2(a.v[1], a.v[3], u, f);
      o.v[2] = clamped_glu2(b.v[0], b.v[2], u, f);
      o.v[3] = clamped_glu2(b.v[1], b.v[3], u, f);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) o.v[e] = clamped_glu2(a.v[e], b.v[e], u, f);
    }
    *reinterpret_cast<bf16x8*>(out + row * ldo + i) = o;
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

// f32: 1 = activations and tables fp32, 0 = bf16. out [rows][S][H]; pos and freq may be null.
int ve_embed_rows(const void* ids, const void* table, const void* pos, const void* freq, void* out, int rows, int H, int vocab, int S, float scale, int f32,
                  cudaStream_t st) {
  if (rows <= 0) return 0;
  if (S < 1 || (freq && !pos)) return cudaErrorInvalidValue;
#define VE_EM(T) launch_pdl(embed_rows_kernel<T>, dim3(rows), dim3(row_threads(H)), 0, st, (const int*)ids, (const T*)table, (const int*)pos, \
    (const double*)freq, (float*)out, H, vocab, S, scale)
  if (f32) VE_EM(float);
  else VE_EM(__nv_bfloat16);
#undef VE_EM
  VE_CHECK_LAUNCH();
}

// h [rows][S][H] contiguous fp32; part null: the streams stay; out null: only the streams are rewritten.
int ve_stream_norm(void* h, const void* part, long ldp, const void* mix, const void* wout, const void* win, const void* w, void* out, long ldo, int rows,
                   int H, int S, float eps, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (S < 1 || S > kMaxStreams || (part && (!mix || !wout)) || (out && (!win || !w))) return cudaErrorInvalidValue;
  const bool vec = !f32 && S <= 4 && H % 4 == 0 && H <= 8192 && win && (!part || ldp % 4 == 0) && (!out || ldo % 4 == 0) && !((uintptr_t)h & 15) &&
                   !((uintptr_t)part & 7) && !((uintptr_t)w & 15) && !((uintptr_t)out & 7);
#define VE_SN(S_, NV) launch_pdl(stream_norm4_kernel<S_, NV, __nv_bfloat16>, dim3(rows), dim3(256), 0, st, (float*)h, (const __nv_bfloat16*)part, ldp, \
    (const float*)mix, (const float*)wout, (const float*)win, (const float*)w, (__nv_bfloat16*)out, ldo, H, eps)
#define VE_SN_V(S_) do { if (H <= 1024) VE_SN(S_, 1); else if (H <= 2048) VE_SN(S_, 2); else if (H <= 4096) VE_SN(S_, 4); else VE_SN(S_, 8); } while (0)
  if (vec) {
    if (S == 1) VE_SN_V(1);
    else if (S == 2) VE_SN_V(2);
    else if (S == 3) VE_SN_V(3);
    else VE_SN_V(4);
    VE_CHECK_LAUNCH();
  }
#undef VE_SN_V
#undef VE_SN
#define VE_SN(T) launch_pdl(stream_norm_kernel<T>, dim3(rows), dim3(row_threads(H)), 0, st, (float*)h, (const T*)part, ldp, (const float*)mix, \
    (const float*)wout, (const float*)win, (const float*)w, (T*)out, ldo, H, S, eps)
  if (f32) VE_SN(float);
  else VE_SN(__nv_bfloat16);
#undef VE_SN
  VE_CHECK_LAUNCH();
}

// h [rows][H] contiguous fp32 += RMS norm of the result * wa (wa null: the result as it is; part null: no result); out = h, or its RMS norm * wo
// (null: not normed; out null: no output). top > 0: a row's result is the sum of rw [rows][top] (null: all one) times rows inv [rows][top]
// (null: in order) of part.
int ve_residual_norm(void* h, const void* part, long ldp, const void* inv, const void* rw, int top, const void* wa, const void* wo, void* out, long ldo, int rows,
                     int H, float eps, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (H < 1 || top < 0 || (wa && !part) || (!part && !out)) return cudaErrorInvalidValue;
  const ResultRows rr{(const int*)inv, (const float*)rw, part ? top : 0};
  const bool vec = !f32 && H % 4 == 0 && H <= 8192 && ldp % 4 == 0 && ldo % 4 == 0 && !(((uintptr_t)h | (uintptr_t)wa | (uintptr_t)wo) & 15) &&
                   !(((uintptr_t)part | (uintptr_t)out) & 7);
  if (f32) launch_pdl(residual_norm_kernel<float>, dim3(rows), dim3(256), 0, st, (float*)h, (const float*)part, ldp, rr, (const float*)wa, (const float*)wo,
                      (float*)out, ldo, H, eps);
  else if (!vec) launch_pdl(residual_norm_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, st, (float*)h, (const __nv_bfloat16*)part, ldp, rr, (const float*)wa,
                            (const float*)wo, (__nv_bfloat16*)out, ldo, H, eps);
#define VE_RN(NV) launch_pdl(residual_norm4_kernel<NV, __nv_bfloat16>, dim3(rows), dim3(256), 0, st, (float*)h, (const __nv_bfloat16*)part, ldp, rr, \
    (const float*)wa, (const float*)wo, (__nv_bfloat16*)out, ldo, H, eps)
  else if (H <= 1024) VE_RN(1);
  else if (H <= 2048) VE_RN(2);
  else if (H <= 4096) VE_RN(4);
  else VE_RN(8);
#undef VE_RN
  VE_CHECK_LAUNCH();
}

int ve_soft_cap(void* x, long n, float cap, cudaStream_t st) {
  if (n <= 0) return 0;
  if (!(cap > 0.f)) return cudaErrorInvalidValue;
  const long blocks = (n + 255) / 256;
  launch_pdl(soft_cap_kernel, dim3((unsigned)(blocks < 148 * 8 ? blocks : 148 * 8)), dim3(256), 0, st, (float*)x, n, cap);
  VE_CHECK_LAUNCH();
}

// z rows [gate F | up F] (blk 0) or blocks of [4 gate | 4 up] (F a multiple of 4); fp32 when x32, else of the activation type. w (null:
// none): row r is first multiplied with w[index[r]].
int ve_clamped_glu(const void* z, long ldz, int x32, void* out, long ldo, int rows, int F, int blk, float alpha, float limit, float shift, const void* w,
                   const void* index, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const Glu u{alpha, limit, shift};
  const RowBy by{(const float*)w, (const int*)index};
  if (F < 1 || (blk && F % 4) || (w && !index)) return cudaErrorInvalidValue;
  const bool vec = !f32 && !x32 && F % 8 == 0 && ldz % 8 == 0 && ldo % 8 == 0 && !((uintptr_t)z & 15) && !((uintptr_t)out & 15);
  const long total = (long)rows * F / (vec ? 8 : 1), blocks = (total + 255) / 256;
  const dim3 grid((unsigned)(blocks < 148 * 8 ? blocks : 148 * 8));
  if (vec) {
    launch_pdl(clamped_glu8_kernel, grid, dim3(256), 0, st, (const __nv_bfloat16*)z, ldz, (__nv_bfloat16*)out, ldo, total, F, blk, u, by);
    VE_CHECK_LAUNCH();
  }
#define VE_CG(X, T) launch_pdl(clamped_glu_kernel<X, T>, grid, dim3(256), 0, st, (const X*)z, ldz, (T*)out, ldo, total, F, blk, u, by)
  if (f32) VE_CG(float, float);
  else if (x32) VE_CG(float, __nv_bfloat16);
  else VE_CG(__nv_bfloat16, __nv_bfloat16);
#undef VE_CG
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

// x (and gate) fp32 when x32, else of the activation type; cols = groups * G. silu: the gate's activation is SiLU, else sigmoid.
int ve_group_rms(const void* x, long ldx, int x32, const void* w, int wlen, const void* gate, long ldg, int silu, void* out, long ldo, int rows, int cols,
                 int G, float eps, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (G <= 0 || cols % G || wlen <= 0) return cudaErrorInvalidValue;
  const int xa = x32 || f32 ? 15 : 7, oa = f32 ? 15 : 7;
  const bool vec = G <= 512 && G % 4 == 0 && wlen % 4 == 0 && ldx % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 && !((uintptr_t)x & xa) && !((uintptr_t)gate & xa) &&
                   !((uintptr_t)out & oa) && !((uintptr_t)w & 15);
  const long groups = (long)rows * (cols / G), blocks = (groups + 7) / 8;
  const dim3 grid(rows, cols / G), block(row_threads(G)), grid4((unsigned)(blocks < 148 * 16 ? blocks : 148 * 16));
#define VE_GR4(N4, X, T) launch_pdl(group_rms4_kernel<N4, X, T>, grid4, dim3(256), 0, st, (const X*)x, ldx, (const float*)w, wlen, (const X*)gate, ldg, silu, \
    (T*)out, ldo, G, cols / G, groups, eps)
#define VE_GR(X, T) do { if (vec && G <= 128) VE_GR4(1, X, T); else if (vec) VE_GR4(4, X, T); \
    else launch_pdl(group_rms_kernel<X, T>, grid, block, 0, st, (const X*)x, ldx, (const float*)w, wlen, (const X*)gate, ldg, silu, (T*)out, ldo, G, eps); } while (0)
  if (f32) VE_GR(float, float);
  else if (x32) VE_GR(float, __nv_bfloat16);
  else VE_GR(__nv_bfloat16, __nv_bfloat16);
#undef VE_GR
#undef VE_GR4
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
