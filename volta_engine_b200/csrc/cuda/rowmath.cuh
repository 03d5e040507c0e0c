// Element formulas shared by the row operators (rowops.cu) and by the decode linears that apply them in their prologue
// (gemv_rows.cu), so that the fused and the separate form of a step agree. Everything in fp32.
#pragma once
#include "common.cuh"

namespace ve {

VE_DEVINL float to_f(float v) { return v; }
VE_DEVINL float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> VE_DEVINL T from_f(float v);
template <> VE_DEVINL float from_f<float>(float v) { return v; }
template <> VE_DEVINL __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

VE_DEVINL float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
VE_DEVINL float4 load4(const __nv_bfloat16* p) {
  const uint2 t = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(t.x << 16), __uint_as_float(t.x & 0xffff0000u), __uint_as_float(t.y << 16), __uint_as_float(t.y & 0xffff0000u));
}
VE_DEVINL void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
VE_DEVINL void store4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

VE_DEVINL float sigmoid_of(float z) { return 1.f / (1.f + expf(-z)); }
VE_DEVINL float silu_of(float z) { return z / (1.f + expf(-z)); }
VE_DEVINL float dyt_of(float h, float alpha, float w, float b) { return fmaf(tanhf(alpha * h), w, b); }

// Gated unit with both halves clamped: min(g, limit) sigmoid(alpha min(g, limit)) (clamp(u, -limit, limit) + shift).
// alpha 1, an infinite limit and shift 0 make it silu(g) u.
struct Glu { float alpha, limit, shift; };
VE_DEVINL float clamped_glu_of(float g, float u, const Glu& c) {
  const float a = fminf(g, c.limit), b = fminf(fmaxf(u, -c.limit), c.limit);
  return a / (1.f + expf(-c.alpha * a)) * (b + c.shift);
}

VE_DEVINL float soft_cap_of(float v, float cap) { return cap * tanhf(v / cap); }

// Sine and cosine (times mul) of a position's angles, by the threads of a block into shared memory. freq: half turns per position, in
// double; the angle is reduced to one turn before it is rounded.
constexpr int kMaxPairs = 256;
VE_DEVINL void angle_row(int pos, const double* __restrict__ freq, int pairs, float mul, float* cs, float* sn) {
  for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
    const double t = (double)pos * freq[i];
    float s, c;
    sincospif((float)(t - 2.0 * rint(0.5 * t)), &s, &c);
    cs[i] = c * mul;
    sn[i] = s * mul;
  }
}

// Residual streams (at most kMaxStreams copies of a row): every stream anew from all old ones and a sublayer's result,
// x_t <- sum_s mix[s][t] x_s + out[t] y; and what a sublayer reads, sum_s in[s] x_s.
constexpr int kMaxStreams = 8;
VE_DEVINL void streams_write(float* x, int S, const float* __restrict__ mix, const float* __restrict__ out, float y) {
  float o[kMaxStreams];
#pragma unroll
  for (int s = 0; s < kMaxStreams; ++s) o[s] = s < S ? x[s] : 0.f;
#pragma unroll
  for (int t = 0; t < kMaxStreams; ++t)
    if (t < S) {
      float v = out[t] * y;
#pragma unroll
      for (int s = 0; s < kMaxStreams; ++s)
        if (s < S) v = fmaf(mix[s * S + t], o[s], v);
      x[t] = v;
    }
}

// PolyNorm: sums of z^2, z^4, z^6 over a row, then c0 z / rms(z) + c1 z^2 / rms(z^2) + c2 z^3 / rms(z^3) + c3
VE_DEVINL void poly_sums(float z, float& s1, float& s2, float& s3) {
  const float q = z * z, q2 = q * q;
  s1 += q;
  s2 += q2;
  s3 = fmaf(q2, q, s3);
}
struct PolyScale { float a1, a2, a3, a0; };
VE_DEVINL PolyScale poly_scale(float s1, float s2, float s3, int n, float eps, const float* __restrict__ coef) {
  const float r = 1.f / (float)n;
  PolyScale p;
  p.a1 = coef[0] / sqrtf(s1 * r + eps);
  p.a2 = coef[1] / sqrtf(s2 * r + eps);
  p.a3 = coef[2] / sqrtf(s3 * r + eps);
  p.a0 = coef[3];
  return p;
}
VE_DEVINL float poly_of(float z, const PolyScale& p) { return fmaf(z, fmaf(z, fmaf(z, p.a3, p.a2), p.a1), p.a0); }

}  // namespace ve
