// Grouped-query softmax attention with its sizes and its score terms as parameters: query / key width and value width may differ and
// need not be powers of two; optional rotary positions and RMS norm (with or without a weight, behind the rotation or in front of it) of
// queries and keys, query temperature by position, a factor per query head, a soft cap of the scores, a sliding window (with or without the
// first tokens of the sequence in sight), bias by distance (a table per head whose last entry holds for everything farther), a sink (one
// more term of the denominator), a factor on the result, a sigmoid gate on every element of it. Values may be rotated by their position
// too: they are cached so, and the result is turned back by the query's position.
//
// Cache: a page of the pool is 64 tokens x row width; this layer sees it as [kv heads][64][kw] (values [kv heads][64][vw]) with kw, vw the
// widths rounded up to 8 elements (pad columns are zero), so layers of unlike sizes share one pool.
//   gqa_store    rotation, norms, temperature, queries as rows [heads][kw], keys and values into the cache
//   gqa_rows     one CTA per (row, head) on the CUDA cores: the all-32-bit form, and sizes outside the range of the others
//   gqa_decode   decode rows: 16 query heads of a kv head x 64-key pages (TMA) on mma.sync, key splits over the grid, the split
//                that ends last merges
//   gqa_prefill  prompt rows on tcgen05 (gqa_tc.cuh)
// Scores, weights and sums are fp32; where weights enter a tensor core they do so as two bf16 terms. No fast-math in this file.
#include "rowmath.cuh"
#include "tmap.h"
#include <float.h>
#include <limits.h>

namespace ve {

constexpr int kGPage = 64;
constexpr int kGMinPages = 2;     // of a key split
constexpr float kLog2e = 1.4426950408889634f;

struct GqaDims {
  int H, G, d, dv, kw, vw;        // query / kv heads, query-key and value widths, cached widths
  long kps, vps;                  // elements per page of the key and the value pool
};
struct GqaScore {
  float scale;
  const float* bias; int L;       // [H][L] by distance, entry L - 1 for everything from L - 1 on (null: none)
  const float* sink;              // [H] (null: none)
  float out_scale;
  int window;                     // keys at distances below it are seen (INT_MAX: all in front)
  const void* gate; long ldg;     // [rows][H dv] (null: none), fp32 (gate32) or bf16
  int gate32, gatev;              // gatev: eight columns from a multiple of eight on are 16-byte aligned
  int keep;                       // keys at positions below it are seen at any distance
  float cap;                      // > 0: scores are cap tanh(score / cap), in front of the bias
  const float2* back; int bpairs; // [rows][bpairs] cosines and sines that the result is turned back by (null: not turned)
  int bneigh;                     // pairs are columns (2 i, 2 i + 1), else (i, i + bpairs)
};
struct GqaTurn {
  const double* freq;             // half turns per position
  int pairs;                      // 0: no rotation
  float mul;
  int neighbours;                 // pairs are columns (2 i, 2 i + 1), else (i, i + pairs)
  const double* vfreq; int vpairs;     // of the values (0: not turned), pairs as above
  float2* back;                   // [rows][vpairs]: cosine and sine of the values' angles (null: not stored)
};
VE_DEVINL float gate_at(const GqaScore& sc, long row, int c) {
  if (!sc.gate) return 1.f;
  const long at = row * sc.ldg + c;
  return sigmoid_of(sc.gate32 ? reinterpret_cast<const float*>(sc.gate)[at] : to_f(reinterpret_cast<const __nv_bfloat16*>(sc.gate)[at]));
}
struct GqaRows {
  const int* pos; const int* slot; const int* page_table;
  int max_pages;
};

// Column c of a result turned back, from it and the other column of its pair.
VE_DEVINL int back_partner(const GqaScore& sc, int c) { return sc.bneigh ? c ^ 1 : c < sc.bpairs ? c + sc.bpairs : c - sc.bpairs; }
VE_DEVINL float turned_back(const GqaScore& sc, long row, int c, float own, float other) {
  const float2 a = sc.back[row * sc.bpairs + (sc.bneigh ? c >> 1 : c < sc.bpairs ? c : c - sc.bpairs)];
  const bool low = sc.bneigh ? !(c & 1) : c < sc.bpairs;
  return fmaf(own, a.x, low ? other * a.y : -(other * a.y));
}
// Four neighbouring columns (from a multiple of four on) whose pairs are neighbours.
VE_DEVINL float4 turned_back4(const GqaScore& sc, long row, int c, float4 v) {
  const float2 a = sc.back[row * sc.bpairs + (c >> 1)], b = sc.back[row * sc.bpairs + (c >> 1) + 1];
  return make_float4(fmaf(v.x, a.x, v.y * a.y), fmaf(v.y, a.x, -(v.x * a.y)), fmaf(v.z, b.x, v.w * b.y), fmaf(v.w, b.x, -(v.z * b.y)));
}

// Pages of a row or a tile: those of the first tokens, then those from the first window on.
struct GqaPages {
  int front, from;                // pages 0 .. front - 1, then from, from + 1, ...
  VE_DEVINL GqaPages(const GqaScore& sc, int pos) : from(max(0, pos - sc.window + 1) / kGPage) { front = min(from, (sc.keep + kGPage - 1) / kGPage); }
  VE_DEVINL int of(int i) const { return i < front ? i : from + i - front; }
  VE_DEVINL int count(int last) const { return front + last / kGPage + 1 - from; }      // last: the last position that is seen
};
VE_DEVINL bool sees(const GqaScore& sc, int dist, int key) { return (unsigned)dist < (unsigned)sc.window || (key < sc.keep && dist >= 0); }

VE_DEVINL int page_of(const GqaRows& r, int slot, int kt) { return r.page_table[(long)slot * r.max_pages + kt]; }

// proj row: [q (H d) | k (G d) | v (G dv) | ...]. grid (rows, ceil((H + 2 G) / 8)), a warp per head. norm: queries and keys are divided by
// their root mean square, times wq / wk where given, behind the rotation (1) or in front of it (2). hmul: factors of the query heads.
template <typename X, typename T>
__global__ void __launch_bounds__(256) gqa_store_kernel(const GqaDims n, const GqaRows rw, const X* __restrict__ proj, long ld, const GqaTurn tn, int norm,
                                                        const float* __restrict__ wq, const float* __restrict__ wk, float eps, float coef, int every,
                                                        const float* __restrict__ hmul, int vec,
                                                        T* __restrict__ qo, T* __restrict__ kpool, T* __restrict__ vpool) {
  __shared__ __align__(16) float qcs[kMaxPairs], qsn[kMaxPairs], vcs[kMaxPairs], vsn[kMaxPairs];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  const int item = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int p = rw.pos[row], s = rw.slot[row];
  if (tn.pairs) angle_row(p, tn.freq, tn.pairs, tn.mul, qcs, qsn);
  if (tn.vpairs) angle_row(p, tn.vfreq, tn.vpairs, 1.f, vcs, vsn);
  if (tn.pairs | tn.vpairs) __syncthreads();
  if (tn.back && blockIdx.y == 0)
    for (int i = threadIdx.x; i < tn.vpairs; i += 256) tn.back[row * tn.vpairs + i] = make_float2(vcs[i], vsn[i]);
  if (item >= n.H + 2 * n.G) return;
  const bool is_q = item < n.H, is_v = item >= n.H + n.G;
  if (s < 0 && !is_q) return;
  const X* src = proj + row * ld + (is_v ? (long)(n.H + n.G) * n.d + (long)(item - n.H - n.G) * n.dv : (long)item * n.d);
  T* dst;
  if (is_q) dst = qo + (row * n.H + item) * n.kw;
  else {
    const int page = page_of(rw, s, p / kGPage), at = p % kGPage;
    dst = is_v ? vpool + page * n.vps + ((long)(item - n.H - n.G) * kGPage + at) * n.vw : kpool + page * n.kps + ((long)(item - n.H) * kGPage + at) * n.kw;
  }
  const int w = is_v ? n.dv : n.d, wide = is_v ? n.vw : n.kw, pairs = is_v ? tn.vpairs : tn.pairs, turned = 2 * pairs;
  const float *cs = is_v ? vcs : qcs, *sn = is_v ? vsn : qsn;
  const float* wn = is_v ? nullptr : is_q ? wq : wk;
  const bool nrm = norm && !is_v, before = nrm && norm == 2;
  float t = is_q && every > 0 ? 1.f + coef * logf((float)((p + 1) / every + 1)) : 1.f;
  if (is_q && hmul) t *= hmul[item];
  if (vec) {                                // widths up to 256 in multiples of eight: four columns per lane and step, kept in registers
    float4 v[2];
    float ss = 0.f, f = 1.f;
    auto normed = [&](float4 x, int i) {    // columns from i on, normed in front of the rotation
      if (!before) return x;
      const float4 q = wn ? *reinterpret_cast<const float4*>(wn + i) : make_float4(1.f, 1.f, 1.f, 1.f);
      return make_float4(x.x * f * q.x, x.y * f * q.y, x.z * f * q.z, x.w * f * q.w);
    };
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = (j * 32 + lane) * 4;
      v[j] = i < w ? load4(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    }
    if (before) f = 1.f / sqrtf(warp_sum(ss) / (float)w + eps);
    ss = 0.f;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = (j * 32 + lane) * 4;
      if (i < w) v[j] = normed(v[j], i);
      if (i < turned) {
        if (tn.neighbours) {
          const float2 c = *reinterpret_cast<const float2*>(cs + i / 2), z = *reinterpret_cast<const float2*>(sn + i / 2);
          v[j] = make_float4(fmaf(v[j].x, c.x, -(v[j].y * z.x)), fmaf(v[j].y, c.x, v[j].x * z.x), fmaf(v[j].z, c.y, -(v[j].w * z.y)),
                             fmaf(v[j].w, c.y, v[j].z * z.y));
        } else {
          const bool low = i < pairs;
          const int k = low ? i : i - pairs, other = low ? i + pairs : k;
          const float4 c = *reinterpret_cast<const float4*>(cs + k), o = normed(load4(src + other), other);
          float4 z = *reinterpret_cast<const float4*>(sn + k);
          if (low) z = make_float4(-z.x, -z.y, -z.z, -z.w);
          v[j] = make_float4(fmaf(v[j].x, c.x, o.x * z.x), fmaf(v[j].y, c.y, o.y * z.y), fmaf(v[j].z, c.z, o.z * z.z), fmaf(v[j].w, c.w, o.w * z.w));
        }
      }
      ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    }
    const float g = nrm && !before ? t / sqrtf(warp_sum(ss) / (float)w + eps) : t;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = (j * 32 + lane) * 4;
      if (i >= w) continue;
      const float4 q = wn && !before ? *reinterpret_cast<const float4*>(wn + i) : make_float4(1.f, 1.f, 1.f, 1.f);
      store4(dst + i, make_float4(v[j].x * g * q.x, v[j].y * g * q.y, v[j].z * g * q.z, v[j].w * g * q.w));
    }
    return;
  }
  float f = 1.f;
  auto raw = [&](int i) { return before ? to_f(src[i]) * f * (wn ? wn[i] : 1.f) : to_f(src[i]); };
  auto value = [&](int i) {
    const float v = raw(i);
    if (i >= turned) return v;
    const bool low = tn.neighbours ? !(i & 1) : i < pairs;
    const int k = tn.neighbours ? i >> 1 : low ? i : i - pairs, other = tn.neighbours ? i ^ 1 : low ? i + pairs : k;
    const float o = raw(other) * sn[k];
    return fmaf(v, cs[k], low ? -o : o);
  };
  if (nrm) {
    float ss = 0.f;
    for (int i = lane; i < w; i += 32) {
      const float v = before ? to_f(src[i]) : value(i);
      ss = fmaf(v, v, ss);
    }
    f = 1.f / sqrtf(warp_sum(ss) / (float)w + eps);
  }
  for (int i = lane; i < wide; i += 32) {
    float v = 0.f;
    if (i < w) {
      v = value(i);
      if (!before) {
        v *= f;
        if (wn) v *= wn[i];
      }
      v *= t;
    }
    dst[i] = from_f<T>(v);
  }
}

// grid (rows, H), 128 threads: warp w takes keys w, w + 4, ...; lane = column mod 32. NC = value columns per lane.
template <int NC, typename T, typename O>
__global__ void __launch_bounds__(128) gqa_rows_kernel(const GqaDims n, const GqaRows rw, const GqaScore sc, const T* __restrict__ q, const T* __restrict__ kpool,
                                                       const T* __restrict__ vpool, O* __restrict__ out, long ldo) {
  extern __shared__ float sm[];             // [kw] query, then [4][NC * 32] outputs
  __shared__ float sm_m[4], sm_l[4];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  const int h = blockIdx.y, g = h / (n.H / n.G), lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int s = rw.slot[row], p = rw.pos[row];
  O* orow = out + row * ldo + (long)h * n.dv;
  if (s < 0) {
    for (int i = threadIdx.x; i < n.dv; i += 128) orow[i] = from_f<O>(0.f);
    return;
  }
  for (int i = threadIdx.x; i < n.kw; i += 128) sm[i] = to_f(q[(row * n.H + h) * n.kw + i]);
  __syncthreads();
  float acc[NC], m = -FLT_MAX, l = 0.f;
#pragma unroll
  for (int j = 0; j < NC; ++j) acc[j] = 0.f;
  const int begin = max(0, p - sc.window + 1), front = min(sc.keep, begin), total = front + p + 1 - begin;      // first tokens, then the window
  for (int i = warp; i < total; i += 4) {
    const int key = i < front ? i : begin + i - front;
    const int page = page_of(rw, s, key / kGPage);
    const T* kr = kpool + page * n.kps + ((long)g * kGPage + key % kGPage) * n.kw;
    const T* vr = vpool + page * n.vps + ((long)g * kGPage + key % kGPage) * n.vw;
    float dot = 0.f, v[NC];
#pragma unroll
    for (int j = 0; j < NC; ++j) v[j] = j * 32 + lane < n.dv ? to_f(vr[j * 32 + lane]) : 0.f;
    for (int i = lane; i < n.d; i += 32) dot = fmaf(to_f(kr[i]), sm[i], dot);
    dot = warp_sum(dot) * sc.scale;
    if (sc.cap > 0.f) dot = soft_cap_of(dot, sc.cap);
    if (sc.bias) dot += sc.bias[(long)h * sc.L + min(p - key, sc.L - 1)];
    const float mn = fmaxf(m, dot), corr = m == -FLT_MAX ? 0.f : expf(m - mn), e = expf(dot - mn);
    m = mn;
    l = fmaf(l, corr, e);
#pragma unroll
    for (int j = 0; j < NC; ++j) acc[j] = fmaf(acc[j], corr, e * v[j]);
  }
  float* os = sm + n.kw;
#pragma unroll
  for (int j = 0; j < NC; ++j) os[warp * NC * 32 + j * 32 + lane] = acc[j];
  if (lane == 0) {
    sm_m[warp] = m;
    sm_l[warp] = l;
  }
  __syncthreads();
  const float snk = sc.sink ? sc.sink[h] : -FLT_MAX;
  const float mx = fmaxf(snk, fmaxf(fmaxf(sm_m[0], sm_m[1]), fmaxf(sm_m[2], sm_m[3])));
  float f[4], lt = sc.sink ? expf(snk - mx) : 0.f;
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    f[w] = sm_m[w] == -FLT_MAX ? 0.f : expf(sm_m[w] - mx);
    lt += sm_l[w] * f[w];
  }
  auto sum = [&](int i) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) v += os[w * NC * 32 + i] * f[w];
    return v / lt;
  };
  for (int i = threadIdx.x; i < n.dv; i += 128) {
    float v = sum(i);
    if (sc.back) v = turned_back(sc, row, i, v, sum(back_partner(sc, i)));
    orow[i] = from_f<O>(v * sc.out_scale * gate_at(sc, row, h * n.dv + i));
  }
}

VE_DEVINL void gq_ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
VE_DEVINL void gq_ldsm_x4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
VE_DEVINL void gq_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
VE_DEVINL uint32_t gq_pack(float lo, float hi) {
  const __nv_bfloat162 t = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&t);
}

// Four columns (from a multiple of four on; c counts over all heads) of an output row of any alignment.
template <typename O>
VE_DEVINL void put_row(O* p, float4 v, const GqaScore& sc, long row, int c, int dv) {
  if (sc.back) v = turned_back4(sc, row, c % dv, v);
  p[0] = from_f<O>(v.x * gate_at(sc, row, c));
  p[1] = from_f<O>(v.y * gate_at(sc, row, c + 1));
  p[2] = from_f<O>(v.z * gate_at(sc, row, c + 2));
  p[3] = from_f<O>(v.w * gate_at(sc, row, c + 3));
}

struct GqaDecode {
  GqaDims n;
  GqaRows rw;
  GqaScore sc;
  const __nv_bfloat16* q;         // [rows][H][kw]
  float* o_part;                  // [rows][H][nsplit][dv]
  float* lse;                     // [rows][H][nsplit], log2 units
  int* tickets;                   // [rows * groups * G], zero between launches
  int nsplit, groups;             // groups of at most 16 query heads of a kv head
  int nst;                        // page stages
  int* status;
};

// grid (rows * groups, G, nsplit), 128 threads. A page is scored by four warps, 16 keys each; their states meet in shared memory.
template <int DQC, int DVC, typename O>
__global__ void __launch_bounds__(128) gqa_decode_kernel(const GqaDecode a, O* __restrict__ out, long ldo, const __grid_constant__ CUtensorMap kmap,
                                                         const __grid_constant__ CUtensorMap vmap) {
  constexpr int KB = DQC * 8192, VB = DVC * 8192, STG = KB + VB, DV = DVC * 64;
  extern __shared__ uint8_t gq_smem[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(gq_smem) + 1023) & ~(uintptr_t)1023);
  __shared__ uint64_t full[4];
  __shared__ int s_last;
  grid_dep_wait();
  grid_dep_launch();
  const GqaDims& n = a.n;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const long row = blockIdx.x / a.groups;
  const int kvh = blockIdx.y, z = blockIdx.z, hpg = n.H / n.G, hg = blockIdx.x % a.groups;
  const int h0 = kvh * hpg + hg * 16, nh = min(16, hpg - hg * 16);
  const int s = a.rw.slot[row];
  if (s < 0) {
    if (z == 0)
      for (int i = tid; i < nh * n.dv; i += 128) out[row * ldo + (long)h0 * n.dv + i] = from_f<O>(0.f);
    return;
  }
  // the grid does not know the position: a row takes as many of its splits as have at least kGMinPages pages
  const int p = a.rw.pos[row];
  const GqaPages pg(a.sc, p);
  const int pages = pg.count(p);
  const int per = max(kGMinPages, (pages + a.nsplit - 1) / a.nsplit), used = (pages + per - 1) / per;
  if (z >= used) return;
  const int kt_begin = z * per, kt_end = min(pages, kt_begin + per);      // (places in the list of pages)
  if (tid == 0) {
    for (int i = 0; i < 4; ++i) mbar_init(&full[i], 1);
    mbar_fence_init();
  }
  __syncthreads();
  auto issue = [&](int kt, int stage) {
    const int page = page_of(a.rw, s, pg.of(kt));
    uint8_t* kb = smem + stage * STG;
    mbar_expect_tx(&full[stage], STG);
#pragma unroll
    for (int c = 0; c < DQC; ++c) tma_load_3d(kb + c * 8192, &kmap, &full[stage], c * 64, kvh * kGPage, page);
#pragma unroll
    for (int c = 0; c < DVC; ++c) tma_load_3d(kb + KB + c * 8192, &vmap, &full[stage], c * 64, kvh * kGPage, page);
  };
  if (tid == 0)
    for (int i = 0; i < a.nst - 1 && kt_begin + i < kt_end; ++i) issue(kt_begin + i, i);
  const bool ok0 = g < nh, ok1 = g + 8 < nh;
  const int head[2] = {h0 + (ok0 ? g : 0), h0 + (ok1 ? g + 8 : 0)};
  uint32_t qf[DQC * 4][4];
#pragma unroll
  for (int kk = 0; kk < DQC * 4; ++kk)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const __nv_bfloat16* qr = a.q + (row * n.H + head[e]) * n.kw;
      const int c = kk * 16 + 2 * t;
      const bool ok = e ? ok1 : ok0;
      qf[kk][e] = ok && c < n.kw ? *reinterpret_cast<const uint32_t*>(qr + c) : 0u;
      qf[kk][2 + e] = ok && c + 8 < n.kw ? *reinterpret_cast<const uint32_t*>(qr + c + 8) : 0u;
    }
  const float scale2 = a.sc.scale * kLog2e, cap2 = a.sc.cap * kLog2e, to_cap = a.sc.cap > 0.f ? a.sc.scale / a.sc.cap : 0.f;
  const float* tab[2] = {a.sc.bias + (long)head[0] * a.sc.L, a.sc.bias + (long)head[1] * a.sc.L};
  float far[2] = {0.f, 0.f};
  if (a.sc.bias) {
    far[0] = tab[0][a.sc.L - 1] * kLog2e;
    far[1] = tab[1][a.sc.L - 1] * kLog2e;
  }
  float o[DVC * 8][4];
#pragma unroll
  for (int i = 0; i < DVC * 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-FLT_MAX, -FLT_MAX}, l_run[2] = {0.f, 0.f};
  const uint32_t base = smem_u32(smem);
  bool failed = false;
  const int mi = lane >> 3, rr = lane & 7, key0 = warp * 16;
  for (int kt = kt_begin; kt < kt_end; ++kt) {
    const int it = kt - kt_begin, stage = it % a.nst;
    const bool ok = mbar_wait(&full[stage], (it / a.nst) & 1);
    if (!__syncthreads_and(ok)) {
      failed = true;
      for (int i = 1; i < a.nst - 1 && kt + i < kt_end; ++i) mbar_wait(&full[(it + i) % a.nst], ((it + i) / a.nst) & 1);   // copies still on their way
      break;
    }
    if (tid == 0 && kt + a.nst - 1 < kt_end) issue(kt + a.nst - 1, (it + a.nst - 1) % a.nst);   // the stage read in the iteration in front
    const uint32_t kb = base + stage * STG, vb = kb + KB;
    float sa[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int kk = 0; kk < DQC * 4; ++kk) {
      const int c = kk >> 2, key = key0 + (mi >> 1) * 8 + rr, ch = (kk & 3) * 2 + (mi & 1);
      uint32_t b0, b1, b2, b3;
      gq_ldsm_x4(kb + c * 8192 + key * 128 + ((ch ^ (key & 7)) << 4), b0, b1, b2, b3);
      gq_mma(sa[0], qf[kk], b0, b1);
      gq_mma(sa[1], qf[kk], b2, b3);
    }
    const int first = pg.of(kt) * kGPage + key0;
    const bool near = a.sc.bias && p - (first + 15) < a.sc.L - 1;
    float mx[2] = {-FLT_MAX, -FLT_MAX};
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int dist = p - (first + nt * 8 + 2 * t + (e & 1)), r = e >> 1;
        const float b = near ? tab[r][min(max(dist, 0), a.sc.L - 1)] * kLog2e : far[r];
        const float x = a.sc.cap > 0.f ? fmaf(tanhf(sa[nt][e] * to_cap), cap2, b) : fmaf(sa[nt][e], scale2, b);
        const float v = sees(a.sc, dist, p - dist) ? x : -FLT_MAX;
        sa[nt][e] = v;
        mx[r] = fmaxf(mx[r], v);
      }
    float corr[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      const float mn = fmaxf(m_run[r], mx[r]);
      corr[r] = m_run[r] == -FLT_MAX ? 0.f : exp2f(m_run[r] - mn);
      m_run[r] = mn;
      l_run[r] *= corr[r];
    }
    uint32_t ph[4], pl[4];                  // weights as A fragments: leading bf16 term and the remainder
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      float pv[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        pv[e] = sa[nt][e] == -FLT_MAX ? 0.f : exp2f(sa[nt][e] - m_run[e >> 1]);
        l_run[e >> 1] += pv[e];
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const uint32_t hi = gq_pack(pv[2 * e], pv[2 * e + 1]);
        ph[nt * 2 + e] = hi;
        pl[nt * 2 + e] = gq_pack(pv[2 * e] - __uint_as_float(hi << 16), pv[2 * e + 1] - __uint_as_float(hi & 0xffff0000u));
      }
    }
#pragma unroll
    for (int i = 0; i < DVC * 8; ++i) {
      o[i][0] *= corr[0];
      o[i][1] *= corr[0];
      o[i][2] *= corr[1];
      o[i][3] *= corr[1];
    }
#pragma unroll
    for (int dp = 0; dp < DVC * 4; ++dp) {
      const int key = key0 + (mi & 1) * 8 + rr, ch = (dp & 3) * 2 + (mi >> 1);
      uint32_t b0, b1, b2, b3;
      gq_ldsm_x4_t(vb + (dp >> 2) * 8192 + key * 128 + ((ch ^ (key & 7)) << 4), b0, b1, b2, b3);
      gq_mma(o[2 * dp], ph, b0, b1);
      gq_mma(o[2 * dp + 1], ph, b2, b3);
      gq_mma(o[2 * dp], pl, b0, b1);
      gq_mma(o[2 * dp + 1], pl, b2, b3);
    }
  }
  if (failed && tid == 0 && a.status) atomicExch(a.status, (int)kErrMbarTimeout);
  __syncthreads();                          // the page buffers are free
  float* ms = reinterpret_cast<float*>(smem);     // [4][16]
  float* ls = ms + 64;                            // [4][16]
  float* os = ls + 64;                            // [4][16][DV]
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    const int hr = g + r * 8;
    if (t == 0) {
      ms[warp * 16 + hr] = m_run[r];
      ls[warp * 16 + hr] = l_run[r];
    }
    if (r ? ok1 : ok0)
#pragma unroll
      for (int i = 0; i < DVC * 8; ++i)
        *reinterpret_cast<float2*>(os + (warp * 16 + hr) * DV + i * 8 + 2 * t) = make_float2(o[i][2 * r], o[i][2 * r + 1]);
  }
  __syncthreads();
  auto sink_of = [&](int h) { return a.sc.sink ? a.sc.sink[h] * kLog2e : -FLT_MAX; };
  for (int i = tid; i < nh * n.dv; i += 128) {
    const int hr = i / n.dv, c = i % n.dv, c2 = a.sc.back && used == 1 ? back_partner(a.sc, c) : c;
    float m = -FLT_MAX, acc = 0.f, acc2 = 0.f, l = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) m = fmaxf(m, ms[w * 16 + hr]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float mw = ms[w * 16 + hr];
      if (mw != -FLT_MAX) {
        const float f = exp2f(mw - m);
        acc = fmaf(os[(w * 16 + hr) * DV + c], f, acc);
        acc2 = fmaf(os[(w * 16 + hr) * DV + c2], f, acc2);
        l = fmaf(ls[w * 16 + hr], f, l);
      }
    }
    if (used == 1) {
      if (a.sc.back) acc = turned_back(a.sc, row, c, acc, acc2);
      const float snk = sink_of(h0 + hr), top = fmaxf(m, snk), f = exp2f(m - top);
      const float den = fmaf(l, f, a.sc.sink ? exp2f(snk - top) : 0.f);
      out[row * ldo + (long)(h0 + hr) * n.dv + c] = from_f<O>(acc * f / den * a.sc.out_scale * gate_at(a.sc, row, (h0 + hr) * n.dv + c));
    } else {
      const long at = (row * n.H + h0 + hr) * a.nsplit + z;
      a.o_part[at * n.dv + c] = l > 0.f ? acc / l : 0.f;
      if (c == 0) a.lse[at] = l > 0.f ? m + log2f(l) : -FLT_MAX;
    }
  }
  if (used == 1) return;
  __threadfence();
  __syncthreads();
  int* tk = a.tickets + (long)blockIdx.x * n.G + kvh;
  if (tid == 0) s_last = atomicAdd(tk, 1) == used - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  // weights of the splits (at most 64) of every head into shared memory, then the weighted sum
  float* sw = ms;                           // [16][64]
  for (int hr = warp; hr < nh; hr += 4) {
    const long at = (row * n.H + h0 + hr) * a.nsplit;
    const float l0 = lane < used ? __ldcg(a.lse + at + lane) : -FLT_MAX, l1 = lane + 32 < used ? __ldcg(a.lse + at + lane + 32) : -FLT_MAX;
    const float snk = sink_of(h0 + hr), top = fmaxf(snk, warp_max(fmaxf(l0, l1)));
    const float w0 = l0 == -FLT_MAX ? 0.f : exp2f(l0 - top), w1 = l1 == -FLT_MAX ? 0.f : exp2f(l1 - top);
    const float den = warp_sum(w0 + w1) + (a.sc.sink ? exp2f(snk - top) : 0.f), inv = a.sc.out_scale / den;
    sw[hr * 64 + lane] = w0 * inv;
    sw[hr * 64 + lane + 32] = w1 * inv;
  }
  __syncthreads();
  if (n.dv % 4 == 0 && (!a.sc.back || a.sc.bneigh)) {
    // four columns per thread; few columns: the splits are dealt to up to four thread groups
    const int c4 = n.dv / 4, items = nh * c4, ng = items <= 32 ? 4 : items <= 64 ? 2 : 1, per = 128 / ng, y0 = tid / per;
    float4* acc4 = reinterpret_cast<float4*>(sw + 16 * 64);
    for (int i = tid % per; i < items; i += per) {
      const int hr = i / c4, c = (i % c4) * 4;
      const float* part = a.o_part + (row * n.H + h0 + hr) * a.nsplit * n.dv + c;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
      for (int y = y0; y < used; y += ng) {
        const float4 x = __ldcg(reinterpret_cast<const float4*>(part + (long)y * n.dv));
        const float f = sw[hr * 64 + y];
        v = make_float4(fmaf(f, x.x, v.x), fmaf(f, x.y, v.y), fmaf(f, x.z, v.z), fmaf(f, x.w, v.w));
      }
      if (ng > 1) acc4[tid] = v;
      else put_row(out + row * ldo + (long)(h0 + hr) * n.dv + c, v, a.sc, row, (h0 + hr) * n.dv + c, n.dv);
    }
    if (ng > 1) {
      __syncthreads();
      if (tid < items) {                    // (at most `per` items)
        float4 v = acc4[tid];
        for (int y = 1; y < ng; ++y) {
          const float4 x = acc4[y * per + tid];
          v = make_float4(v.x + x.x, v.y + x.y, v.z + x.z, v.w + x.w);
        }
        const int c = (h0 + tid / c4) * n.dv + (tid % c4) * 4;
        put_row(out + row * ldo + c, v, a.sc, row, c, n.dv);
      }
    }
  } else {
    for (int i = tid; i < nh * n.dv; i += 128) {
      const int hr = i / n.dv, c = i % n.dv;
      const float* part = a.o_part + (row * n.H + h0 + hr) * a.nsplit * n.dv + c;
      auto sum = [&](int off) {
        float acc = 0.f;
#pragma unroll 8
        for (int y = 0; y < used; ++y) acc = fmaf(sw[hr * 64 + y], __ldcg(part + (long)y * n.dv + off), acc);
        return acc;
      };
      float acc = sum(0);
      if (a.sc.back) acc = turned_back(a.sc, row, c, acc, sum(back_partner(a.sc, c) - c));
      out[row * ldo + (long)(h0 + hr) * n.dv + c] = from_f<O>(acc * gate_at(a.sc, row, (h0 + hr) * n.dv + c));
    }
  }
  if (tid == 0) *tk = 0;
}

template <int DQC, int DVC, typename O>
static int launch_gqa_decode(GqaDecode a, void* out, long ldo, const CUtensorMap& km, const CUtensorMap& vm, int rows, cudaStream_t st) {
  constexpr int stage = (DQC + DVC) * 8192, merge = (128 + 64 * DVC * 64) * 4;
  a.nst = stage * 4 <= 96 * 1024 ? 4 : stage * 3 <= 208 * 1024 ? 3 : 2;
  int smem = a.nst * stage;
  if (smem < merge) smem = merge;
  smem += 1024;
  static bool attr = false;
  if (!attr) {
    const cudaError_t e = cudaFuncSetAttribute(gqa_decode_kernel<DQC, DVC, O>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
    attr = true;
  }
  launch_pdl(gqa_decode_kernel<DQC, DVC, O>, dim3(rows * a.groups, a.n.G, a.nsplit), dim3(128), smem, st, a, (O*)out, ldo, km, vm);
  return (int)cudaGetLastError();
}

}  // namespace ve
#include "gqa_tc.cuh"

using namespace ve;

#define VE_GDIMS int H, int G, int d, int dv, int kw, int vw, long kps, long vps
#define VE_GMAKE GqaDims{H, G, d, dv, kw, vw, kps, vps}
#define VE_GROWS const void* pos, const void* slot, const void* page_table, int max_pages
#define VE_RMAKE GqaRows{(const int*)pos, (const int*)slot, (const int*)page_table, max_pages}
#define VE_GSCORE float scale, const void* bias, int L, const void* sink, float out_scale, int window, const void* gate, long ldg, int gate32, int keep, float cap, \
    const void* back, int bpairs, int bneigh
#define VE_SMAKE gscore(scale, bias, L, sink, out_scale, window, gate, ldg, gate32, dv, keep, cap, back, bpairs, bneigh)
static GqaScore gscore(float scale, const void* bias, int L, const void* sink, float out_scale, int window, const void* gate, long ldg, int gate32, int dv,
                       int keep, float cap, const void* back, int bpairs, int bneigh) {
  return GqaScore{scale, (const float*)bias, L, (const float*)sink, out_scale, window > 0 ? window : INT_MAX, gate, ldg, gate32,
                  dv % 8 == 0 && ldg % 8 == 0 && !((uintptr_t)gate & 15), window > 0 && keep > 0 ? keep : 0, cap, (const float2*)back, bpairs, bneigh};
}
static bool gdims_ok(const GqaDims& n) {
  return n.G > 0 && n.H > 0 && n.H % n.G == 0 && n.d > 0 && n.dv > 0 && n.kw >= n.d && n.vw >= n.dv && n.kps >= (long)n.G * 64 * n.kw && n.vps >= (long)n.G * 64 * n.vw;
}
// A pool as [pages][G * 64][w] with box 64 tokens x 64 columns (columns from w on read as zero).
static int pool_map(CUtensorMap* m, const void* pool, long pages, const GqaDims& n, int w, long ps) {
  return make_tmap_3d(m, pool, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, pages, (uint64_t)n.G * 64, w, (uint64_t)ps * 2, (uint64_t)w * 2, 64, 64,
                      CU_TENSOR_MAP_SWIZZLE_128B);
}

extern "C" {

// proj rows fp32 when x32 (else bf16); f32: queries and pools fp32 (else bf16). pairs 0: no rotation; norm 0: no norm, 1: behind the rotation, 2: in
// front of it, wq and wk are its weights (null: none); every 0: no temperature; hmul: factors of the query heads (null: none); vpairs: 0, or dv / 2
// pairs of value columns, whose angles are stored to back [rows][vpairs][2] (null: not).
int ve_gqa_store(VE_GDIMS, VE_GROWS, const void* proj, long ld, int x32, const void* freq, int pairs, float mul, int neighbours, int norm, const void* wq,
                 const void* wk, float eps, float coef, int every, const void* hmul, const void* vfreq, int vpairs, void* back, void* qo, void* kpool, void* vpool, int rows, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const GqaDims n = VE_GMAKE;
  if (!gdims_ok(n) || pairs < 0 || pairs > kMaxPairs || 2 * pairs > d || (pairs && !freq) || (vpairs && (2 * vpairs != dv || vpairs > kMaxPairs || !vfreq))) return cudaErrorInvalidValue;
  const dim3 grid(rows, (H + 2 * G + 7) / 8);
  const GqaTurn tn{(const double*)freq, pairs, mul, neighbours, (const double*)vfreq, vpairs, (float2*)back};
  const int vec = d % 8 == 0 && dv % 8 == 0 && d <= 256 && dv <= 256 && kw == d && vw == dv && ld % 4 == 0 && !((uintptr_t)proj & 15) && !((uintptr_t)wq & 15) &&
                  !((uintptr_t)wk & 15) && pairs % (neighbours ? 2 : 4) == 0 && vpairs % (neighbours ? 2 : 4) == 0;
#define VE_GS(X, T) launch_pdl(gqa_store_kernel<X, T>, grid, dim3(256), 0, st, n, VE_RMAKE, (const X*)proj, ld, tn, norm, (const float*)wq, (const float*)wk, eps, coef, \
    every, (const float*)hmul, vec, (T*)qo, (T*)kpool, (T*)vpool)
  if (f32) VE_GS(float, float);
  else if (x32) VE_GS(float, __nv_bfloat16);
  else VE_GS(__nv_bfloat16, __nv_bfloat16);
#undef VE_GS
  VE_CHECK_LAUNCH();
}

// o32: fp32 output. d <= 2048, dv <= 1024.
int ve_gqa_rows(VE_GDIMS, VE_GROWS, VE_GSCORE, const void* q, const void* kpool, const void* vpool, void* out, long ldo, int o32, int rows, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const GqaDims n = VE_GMAKE;
  if (!gdims_ok(n) || kw > 2048 || dv > 1024 || (bias && L < 1) || (f32 && !o32) || (back && 2 * bpairs != dv)) return cudaErrorInvalidValue;
#define VE_GR(NC, T, O) launch_pdl(gqa_rows_kernel<NC, T, O>, dim3(rows, H), dim3(128), (size_t)(kw + 4 * NC * 32) * 4, st, n, VE_RMAKE, VE_SMAKE, (const T*)q, \
    (const T*)kpool, (const T*)vpool, (O*)out, ldo)
#define VE_GR_T(T, O) do { if (dv <= 64) VE_GR(2, T, O); else if (dv <= 128) VE_GR(4, T, O); else if (dv <= 256) VE_GR(8, T, O); else VE_GR(32, T, O); } while (0)
  if (f32) VE_GR_T(float, float);
  else if (o32) VE_GR_T(__nv_bfloat16, float);
  else VE_GR_T(__nv_bfloat16, __nv_bfloat16);
#undef VE_GR_T
#undef VE_GR
  VE_CHECK_LAUNCH();
}

// kw and vw multiples of 8, at most 256; nsplit <= 64; groups = ceil(H / G / 16); tickets: rows * groups * G zeros.
int ve_gqa_decode(VE_GDIMS, VE_GROWS, VE_GSCORE, const void* q, const void* kpool, const void* vpool, long pages, void* o_part, void* lse, void* tickets, int nsplit,
                  void* out, long ldo, int o32, int rows, void* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  const GqaDims n = VE_GMAKE;
  if (!gdims_ok(n) || kw % 8 || vw % 8 || kw > 256 || vw > 256 || nsplit < 1 || nsplit > 64 || (bias && L < 1) || (back && 2 * bpairs != dv) || (nsplit > 1 && (!o_part || !lse || !tickets)))
    return cudaErrorInvalidValue;
  CUtensorMap km, vm;
  int rc = pool_map(&km, kpool, pages, n, kw, kps);
  if (!rc) rc = pool_map(&vm, vpool, pages, n, vw, vps);
  if (rc) return rc;
  GqaDecode a{n, VE_RMAKE, VE_SMAKE, (const __nv_bfloat16*)q, (float*)o_part, (float*)lse, (int*)tickets, nsplit, (H / G + 15) / 16, 2, (int*)status};
  const int qc = (kw + 63) / 64, vc = (vw + 63) / 64;
#define VE_GD(Q, V) return o32 ? launch_gqa_decode<Q, V, float>(a, out, ldo, km, vm, rows, st) : launch_gqa_decode<Q, V, __nv_bfloat16>(a, out, ldo, km, vm, rows, st)
#define VE_GD_V(Q) do { if (vc == 1) VE_GD(Q, 1); if (vc == 2) VE_GD(Q, 2); VE_GD(Q, 4); } while (0)
  if (qc == 1) VE_GD_V(1);
  if (qc == 2) VE_GD_V(2);
  VE_GD_V(4);
#undef VE_GD_V
#undef VE_GD
}

// Tiles of at most 128 / (H / G) tokens of one sequence (rows tile_first .. + tile_count of the batch); kw <= 256, vw <= 128, scale > 0, pairs of
// columns that the result is turned back in are neighbours.
int ve_gqa_prefill(VE_GDIMS, VE_GROWS, VE_GSCORE, const void* q, const void* kpool, const void* vpool, long pages, const void* tile_first, const void* tile_count,
                   int ntiles, void* out, long ldo, void* status, cudaStream_t st) {
  if (ntiles <= 0) return 0;
  const GqaDims n = VE_GMAKE;
  if (!gdims_ok(n) || kw % 8 || vw % 8 || kw > 256 || vw > 128 || H / G > 128 || !(scale > 0.f) || ((uintptr_t)q & 15) || (bias && L < 1) ||
      (back && (2 * bpairs != dv || !bneigh))) return cudaErrorInvalidValue;
  CUtensorMap km, vm;
  int rc = pool_map(&km, kpool, pages, n, kw, kps);
  if (!rc) rc = pool_map(&vm, vpool, pages, n, vw, vps);
  if (rc) return rc;
  const int vec = dv % 8 == 0 && ldo % 8 == 0 && !((uintptr_t)out & 15);
  GqaTc p{n, VE_RMAKE, VE_SMAKE, (const __nv_bfloat16*)q, (const int*)tile_first, (const int*)tile_count, (__nv_bfloat16*)out, ldo, vec, (int*)status};
  const int qc = (kw + 63) / 64;
  if (vw <= 64) {
    if (qc == 1) return launch_gqa_tc<1, 1>(p, km, vm, ntiles, st);
    if (qc == 2) return launch_gqa_tc<2, 1>(p, km, vm, ntiles, st);
    return launch_gqa_tc<4, 1>(p, km, vm, ntiles, st);
  }
  if (qc == 1) return launch_gqa_tc<1, 2>(p, km, vm, ntiles, st);
  if (qc == 2) return launch_gqa_tc<2, 2>(p, km, vm, ntiles, st);
  return launch_gqa_tc<4, 2>(p, km, vm, ntiles, st);
}

}  // extern "C"
