// Latent attention with sizes as parameters. Per token and layer the cache holds one row shared by all heads,
//     [ c (kv_rank) | zeros up to rot0 | rotated key part (rot) | zeros ]      (row pitch: the pool's, a multiple of 64)
// with c = RMSNorm of the projected latent. Head h: unrotated key W_uk[h] c, value W_uv[h] c.
//   latent_prep     q rotated in place, cache row written (prompt rows); or, per head, the absorbed query
//                   [ W_uk[h]^T q_un | q_rot ] in the cache row's layout plus the cache row (decode rows)
//   latent_attn     absorbed attention, one CTA per (row, head), any sizes, fp32 arithmetic (all-32-bit form; sizes the
//                   tensor-core kernels do not take). The tensor-core decode kernel is in mla.cu.
//   latent_expand   merges split partials and multiplies by W_uv
//   latent_gather   a sequence's cache rows, contiguous
//   latent_prefill  prompt rows against expanded keys / values: mma.sync flash attention, 64 rows x 64 keys; scores and
//                   weights keep 32-bit quality (weights enter the second product as two bf16 terms). On tcgen05 (latent_tc.cuh)
//                   where plain + rotated width are at most three chunks of 64 columns and the values two, else on mma.sync
// A sliding window hides keys at distances from it on; prompt rows then expand only the cached rows that some row of their portion sees.
// Angles come from a table of half turns per position in double, so they are exact at any position; sine and cosine may carry a factor.
// No fast-math in this file. Neighbouring dimensions (2i, 2i + 1) form a rotation pair.
#include "rowmath.cuh"
#include "tmap.h"
#include <float.h>
#include <limits.h>

namespace ve {

constexpr int kLPage = 64;

struct LatentDims {
  int H, d, rot, dv, kr;     // heads, unrotated / rotated query width, value width, latent width
  int rot0, W, pitch;        // column of the rotated part, row width written by this layer, pool row pitch
};
struct LatentTurn {
  const double* freq;        // half turns per position
  float mul;                 // factor on sine and cosine
};

template <typename K, typename T>
VE_DEVINL void store_latent_row(const LatentDims& n, const K* __restrict__ kv, const float* __restrict__ w, const float* cs, const float* sn,
                                T* __restrict__ dst, float eps, float* red) {
  float ss = 0.f;
  for (int i = threadIdx.x; i < n.kr; i += blockDim.x) {
    const float v = to_f(kv[i]);
    ss = fmaf(v, v, ss);
  }
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)n.kr + eps);
  for (int i = threadIdx.x; i < n.W; i += blockDim.x) {
    float v = 0.f;
    if (i < n.kr) v = to_f(kv[i]) * inv * w[i];
    else if (i >= n.rot0 && i < n.rot0 + n.rot) {
      const int r = i - n.rot0, p = r >> 1;
      const float x = to_f(kv[n.kr + (r & ~1)]), y = to_f(kv[n.kr + (r | 1)]);
      v = (r & 1) ? fmaf(y, cs[p], x * sn[p]) : fmaf(x, cs[p], -(y * sn[p]));
    }
    dst[i] = from_f<T>(v);
  }
}

template <typename T>
VE_DEVINL T* cache_row(T* pool, const LatentDims& n, const int* page_table, int max_pages, int slot, int pos) {
  const int page = page_table[(long)slot * max_pages + pos / kLPage];
  return pool + ((long)page * kLPage + pos % kLPage) * n.pitch;
}

// Prompt rows: grid (rows). q [rows][H (d + rot)] of type X -> qo of type T (may be the same memory when X = T).
template <typename X, typename K, typename T>
__global__ void __launch_bounds__(256) latent_rope_store_kernel(const LatentDims n, const X* q, long ldq, T* qo, long ldqo, const K* __restrict__ kv,
                                                                long ldkv, const float* __restrict__ w, const LatentTurn tn,
                                                                const int* __restrict__ pos, const int* __restrict__ slot,
                                                                const int* __restrict__ page_table, int max_pages, T* __restrict__ pool, float eps) {
  __shared__ float red[33], cs[128], sn[128];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  const int p = pos[row], s = slot[row];
  if (s < 0) return;
  angle_row(p, tn.freq, n.rot / 2, tn.mul, cs, sn);
  __syncthreads();
  const int hw = n.d + n.rot;
  if (qo) {
    if ((const void*)qo == (const void*)q) {
      const int pairs = n.rot / 2;
      for (int i = threadIdx.x; i < n.H * pairs; i += blockDim.x) {
        const int h = i / pairs, j = i % pairs;
        const long c = (long)h * hw + n.d + 2 * j;
        const float x = to_f(q[row * ldq + c]), y = to_f(q[row * ldq + c + 1]);
        qo[row * ldqo + c] = from_f<T>(fmaf(x, cs[j], -(y * sn[j])));
        qo[row * ldqo + c + 1] = from_f<T>(fmaf(y, cs[j], x * sn[j]));
      }
    } else {
      for (int i = threadIdx.x; i < n.H * hw; i += blockDim.x) {
        const int c = i % hw;
        float v = to_f(q[row * ldq + i]);
        if (c >= n.d) {
          const int r = c - n.d, j = r >> 1;
          const float o = to_f(q[row * ldq + (r & 1 ? i - 1 : i + 1)]);
          v = (r & 1) ? fmaf(v, cs[j], o * sn[j]) : fmaf(v, cs[j], -(o * sn[j]));
        }
        qo[row * ldqo + i] = from_f<T>(v);
      }
    }
  }
  store_latent_row(n, kv + row * ldkv, w, cs, sn, cache_row(pool, n, page_table, max_pages, s, p), eps, red);
}

// Decode rows: grid (rows, H + 1, nz). Block y < H: latent columns [z * cols, ...) of head y's absorbed query (z = 0: also the
// rotated part); block y == H (z == 0): the cache row. 128 threads = 16 groups over d x 8 lanes over columns (VEC each).
template <int VEC, typename X, typename K, typename T>
__global__ void __launch_bounds__(128) latent_absorb_kernel(const LatentDims n, const X* __restrict__ q, long ldq, const K* __restrict__ kv, long ldkv,
                                                            const float* __restrict__ w, const T* __restrict__ w_uk, const LatentTurn tn,
                                                            const int* __restrict__ pos, const int* __restrict__ slot,
                                                            const int* __restrict__ page_table, int max_pages, T* __restrict__ pool,
                                                            T* __restrict__ q_abs, int qw, float eps) {
  __shared__ float red[33], cs[128], sn[128], qs[256];
  __shared__ float part[16][8 * VEC];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  const int h = blockIdx.y, z = blockIdx.z, tid = threadIdx.x;
  const int p = pos[row], s = slot[row];
  if (s < 0 || (h == n.H && z > 0)) return;
  if (z == 0) angle_row(p, tn.freq, n.rot / 2, tn.mul, cs, sn);
  if (h == n.H) {
    __syncthreads();
    store_latent_row(n, kv + row * ldkv, w, cs, sn, cache_row(pool, n, page_table, max_pages, s, p), eps, red);
    return;
  }
  const X* qr = q + row * ldq + (long)h * (n.d + n.rot);
  const int grp = tid >> 3, l8 = tid & 7, c0 = (z * 8 + l8) * VEC;
  float acc[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) acc[j] = 0.f;
  for (int d0 = 0; d0 < n.d; d0 += 256) {              // the query in pieces of 256 columns
    const int dn = min(256, n.d - d0);
    __syncthreads();
    for (int i = tid; i < dn; i += 128) qs[i] = to_f(qr[d0 + i]);
    __syncthreads();
    if (c0 < n.kr) {
      const T* wp = w_uk + ((long)h * n.d + d0) * n.kr + c0;
#pragma unroll 4
      for (int i = grp; i < dn; i += 16) {
        T t[VEC];
        if (VEC * sizeof(T) == 16) *reinterpret_cast<uint4*>(t) = *reinterpret_cast<const uint4*>(wp + (long)i * n.kr);
        else
#pragma unroll
          for (int j = 0; j < VEC; ++j) t[j] = wp[(long)i * n.kr + j];
#pragma unroll
        for (int j = 0; j < VEC; ++j) acc[j] = fmaf(qs[i], to_f(t[j]), acc[j]);
      }
    }
  }
#pragma unroll
  for (int j = 0; j < VEC; ++j) part[grp][l8 * VEC + j] = acc[j];
  __syncthreads();
  T* out = q_abs + (row * n.H + h) * (long)qw;
  for (int i = tid; i < 8 * VEC; i += 128) {
    const int c = z * 8 * VEC + i;
    if (c < n.kr) {
      float v = 0.f;
#pragma unroll
      for (int y = 0; y < 16; ++y) v += part[y][i];
      out[c] = from_f<T>(v);
    }
  }
  if (z == 0)
    for (int i = n.kr + tid; i < qw; i += 128) {
      float v = 0.f;
      if (i >= n.rot0 && i < n.rot0 + n.rot) {
        const int r = i - n.rot0, j = r >> 1;
        const float x = to_f(qr[n.d + (r & ~1)]), y = to_f(qr[n.d + (r | 1)]);
        v = (r & 1) ? fmaf(y, cs[j], x * sn[j]) : fmaf(x, cs[j], -(y * sn[j]));
      }
      out[i] = from_f<T>(v);
    }
}

// Absorbed attention on the CUDA cores: grid (rows, H), 128 threads; warp w takes keys w, w + 4, ...; lane = column mod 32.
template <int NC, typename T>
__global__ void __launch_bounds__(128) latent_attn_kernel(const LatentDims n, const T* __restrict__ q_abs, int qw, const int* __restrict__ pos,
                                                          const int* __restrict__ slot, const int* __restrict__ page_table, int max_pages,
                                                          const T* __restrict__ pool, float scale, int window, float* __restrict__ o_lat) {
  extern __shared__ float sm[];             // [qw] query, then [4][NC * 32] outputs
  __shared__ float sm_m[4], sm_l[4];
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  const int h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int s = slot[row], p = pos[row];
  if (s < 0) return;
  for (int i = threadIdx.x; i < qw; i += 128) sm[i] = to_f(q_abs[(row * n.H + h) * (long)qw + i]);
  __syncthreads();
  float acc[NC], m = -FLT_MAX, l = 0.f;
#pragma unroll
  for (int j = 0; j < NC; ++j) acc[j] = 0.f;
  for (int key = max(0, p - window + 1) + warp; key <= p; key += 4) {
    const int page = page_table[(long)s * max_pages + key / kLPage];
    const T* kr = pool + ((long)page * kLPage + key % kLPage) * n.pitch;
    float c[NC], dot = 0.f;
#pragma unroll
    for (int j = 0; j < NC; ++j) {
      const int i = j * 32 + lane;
      c[j] = i < n.kr ? to_f(kr[i]) : 0.f;
      if (i < n.kr) dot = fmaf(c[j], sm[i], dot);
    }
    for (int i = lane; i < n.rot; i += 32) dot = fmaf(to_f(kr[n.rot0 + i]), sm[n.rot0 + i], dot);
    dot = warp_sum(dot) * scale;
    const float mn = fmaxf(m, dot), corr = m == -FLT_MAX ? 0.f : expf(m - mn), e = expf(dot - mn);
    m = mn;
    l = fmaf(l, corr, e);
#pragma unroll
    for (int j = 0; j < NC; ++j) acc[j] = fmaf(acc[j], corr, e * c[j]);
  }
  float* os = sm + qw;
#pragma unroll
  for (int j = 0; j < NC; ++j) os[warp * NC * 32 + j * 32 + lane] = acc[j];
  if (lane == 0) {
    sm_m[warp] = m;
    sm_l[warp] = l;
  }
  __syncthreads();
  const float mx = fmaxf(fmaxf(sm_m[0], sm_m[1]), fmaxf(sm_m[2], sm_m[3]));
  float f[4], lt = 0.f;
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    f[w] = sm_m[w] == -FLT_MAX ? 0.f : expf(sm_m[w] - mx);
    lt += sm_l[w] * f[w];
  }
  for (int i = threadIdx.x; i < n.kr; i += 128) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) v += os[w * NC * 32 + i] * f[w];
    o_lat[(row * n.H + h) * (long)n.kr + i] = v / lt;
  }
}

// out[row][h dv + v] = sum_c o[c] W_uv[h dv + v][c], o = merged split partials (o_part [rows][H][nsplit][ldp], lse in log2
// units; lse null: one finished partial). grid (rows, H, nz), 512 threads: four groups share the splits (every partial's load is
// in flight at once), then a warp per value row. Dynamic shared memory: 4 kr floats.
template <int VEC, typename T>
__global__ void __launch_bounds__(512) latent_expand_kernel(const LatentDims n, const float* __restrict__ o_part, const float* __restrict__ lse,
                                                            int nsplit, int ldp, const T* __restrict__ w_uv, const int* __restrict__ slot,
                                                            T* __restrict__ out, long ldo, int vper) {
  extern __shared__ float os[];                           // [4][kr]
  __shared__ float sw[64], s_inv;
  grid_dep_wait();
  grid_dep_launch();
  const long row = blockIdx.x;
  const int h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, sg = tid >> 7;
  const int v0 = blockIdx.z * vper, v1 = min(n.dv, v0 + vper);
  if (slot[row] < 0) {
    for (int v = v0 + tid; v < v1; v += 512) out[row * ldo + (long)h * n.dv + v] = from_f<T>(0.f);
    return;
  }
  const long base = (row * n.H + h) * nsplit;
  if (lse) {
    if (warp == 0) {                                      // weights of at most 64 splits
      const float l0 = lane < nsplit ? lse[base + lane] : -FLT_MAX, l1 = lane + 32 < nsplit ? lse[base + lane + 32] : -FLT_MAX;
      const float mx = warp_max(fmaxf(l0, l1));
      const float w0 = l0 == -FLT_MAX ? 0.f : exp2f(l0 - mx), w1 = l1 == -FLT_MAX ? 0.f : exp2f(l1 - mx);
      sw[lane] = w0;
      sw[lane + 32] = w1;
      const float ws = warp_sum(w0 + w1);
      if (lane == 0) s_inv = ws > 0.f ? 1.f / ws : 0.f;
    }
    __syncthreads();
    for (int c = tid & 127; c < n.kr; c += 128) {
      float acc = 0.f;
#pragma unroll 16
      for (int i = sg; i < nsplit; i += 4) acc = fmaf(sw[i], sw[i] != 0.f ? o_part[(base + i) * ldp + c] : 0.f, acc);   // (an empty split left nothing)
      os[sg * n.kr + c] = acc;
    }
    __syncthreads();
    const float inv = s_inv;
    for (int c = tid; c < n.kr; c += 512) os[c] = (os[c] + os[n.kr + c] + os[2 * n.kr + c] + os[3 * n.kr + c]) * inv;
  } else {
    for (int c = tid; c < n.kr; c += 512) os[c] = o_part[base * ldp + c];
  }
  __syncthreads();
  for (int v = v0 + warp; v < v1; v += 16) {
    const T* w = w_uv + ((long)h * n.dv + v) * n.kr;
    float acc = 0.f;
#pragma unroll 2
    for (int c = lane * VEC; c < n.kr; c += 32 * VEC) {
      T t[VEC];
      if (VEC * sizeof(T) == 16) *reinterpret_cast<uint4*>(t) = *reinterpret_cast<const uint4*>(w + c);
      else
#pragma unroll
        for (int j = 0; j < VEC; ++j) t[j] = w[c + j];
#pragma unroll
      for (int j = 0; j < VEC; ++j) acc = fmaf(to_f(t[j]), os[c + j], acc);
    }
    acc = warp_sum(acc);
    if (lane == 0) out[row * ldo + (long)h * n.dv + v] = from_f<T>(acc);
  }
}

// rows [0, total) of out [total][W]: cached rows of seg_slot[g] from position seg_start[g] on stand from row seg_base[g] on. 16-byte pieces.
__global__ void latent_gather_kernel(const __nv_bfloat16* __restrict__ pool, int pitch, const int* __restrict__ page_table, int max_pages,
                                     const int* __restrict__ seg_slot, const int* __restrict__ seg_base, const int* __restrict__ seg_start, int nseg,
                                     __nv_bfloat16* __restrict__ out,
                                     int W, int total) {
  grid_dep_wait();
  grid_dep_launch();
  const int per = W / 8;
  for (long i = blockIdx.x * (long)blockDim.x + threadIdx.x; i < (long)total * per; i += (long)gridDim.x * blockDim.x) {
    const int r = (int)(i / per), c = (int)(i % per) * 8;
    int g = 0;
    while (g + 1 < nseg && seg_base[g + 1] <= r) ++g;
    const int key = seg_start[g] + r - seg_base[g];
    const int page = page_table[(long)seg_slot[g] * max_pages + key / kLPage];
    *reinterpret_cast<uint4*>(out + (long)r * W + c) = *reinterpret_cast<const uint4*>(pool + ((long)page * kLPage + key % kLPage) * pitch + c);
  }
}

VE_DEVINL void lp_ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
VE_DEVINL void lp_ldsm_x4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
VE_DEVINL void lp_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
VE_DEVINL uint32_t lp_pack(float lo, float hi) {
  const __nv_bfloat162 t = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&t);
}
VE_DEVINL void cp_async16(uint32_t dst, const void* src, bool in) {      // 16 bytes, zeros when !in (the source is not read then)
  const int n = in ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}

struct LatentPrefill {
  LatentDims n;
  const __nv_bfloat16* q; long ldq;        // [rows][H (d + rot)], rotated
  const __nv_bfloat16* up; long ldu;       // [keys][H d | H dv], expanded from the gathered latents
  const __nv_bfloat16* lat; int W;         // [keys][W], gathered cache rows (the rotated part is read)
  const int* pos;
  const int* tile_first; const int* tile_count; const int* tile_base;   // query tiles; tile_base = first key row of the sequence,
  const int* tile_key0;                    // which is this position
  int window;
  __nv_bfloat16* out; long ldo;            // [rows][H dv]
  float scale_log2;
};

// grid (tiles, H), 128 threads: 64 query rows of one sequence, 16 per warp. DQ, DV: padded widths (multiples of 64).
template <int DQ, int DV>
__global__ void __launch_bounds__(128) latent_prefill_kernel(const LatentPrefill p) {
  constexpr int KP = DQ * 2 + 16, VP = DV * 2 + 16;      // row pitches in bytes (no bank conflicts for ldmatrix)
  constexpr int STAGE = 64 * (KP + VP);
  extern __shared__ __align__(16) uint8_t lsm[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  grid_dep_wait();
  grid_dep_launch();
  const LatentDims& n = p.n;
  const int tile = gridDim.x - 1 - blockIdx.x, h = blockIdx.y;          // late tiles (many keys) first
  const int first = p.tile_first[tile], count = p.tile_count[tile];
  const int win = p.window, skip = max(0, p.pos[first] - win + 1 - p.tile_key0[tile]) / 64 * 64;      // key rows that no row of the tile sees
  const int key0 = p.tile_key0[tile] + skip;
  const long kbase = p.tile_base[tile] + skip;
  const int hw = n.d + n.rot;
  for (int i = tid; i < 2 * STAGE / 16; i += 128) *reinterpret_cast<uint4*>(lsm + i * 16) = make_uint4(0, 0, 0, 0);   // pad columns stay zero
  int r_row[2], r_pos[2];
  bool r_ok[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = warp * 16 + g + e * 8;
    r_ok[e] = r < count;
    r_row[e] = first + (r_ok[e] ? r : 0);
    r_pos[e] = p.pos[r_row[e]];
  }
  const int keys = p.pos[first + count - 1] + 1 - key0, nkt = (keys + 63) / 64;
  uint32_t qf[DQ / 16][4];
#pragma unroll
  for (int kk = 0; kk < DQ / 16; ++kk)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const __nv_bfloat16* qr = p.q + (long)r_row[e] * p.ldq + (long)h * hw;
      const int c = kk * 16 + 2 * t;
      qf[kk][e] = (r_ok[e] && c < hw) ? *reinterpret_cast<const uint32_t*>(qr + c) : 0u;
      qf[kk][2 + e] = (r_ok[e] && c + 8 < hw) ? *reinterpret_cast<const uint32_t*>(qr + c + 8) : 0u;
    }
  __syncthreads();
  const uint32_t sbase = smem_u32(lsm);
  const int kd8 = n.d / 8, kr8 = n.rot / 8, kv8 = n.dv / 8, per = kd8 + kr8 + kv8;
  auto issue = [&](int kt, int stage) {
    const uint32_t kb = sbase + stage * STAGE, vb = kb + 64 * KP;
    for (int i = tid; i < 64 * per; i += 128) {
      const int key = i / per, c = i % per;
      const bool in = kt * 64 + key < keys;
      const long kr = kbase + (in ? kt * 64 + key : 0);
      if (c < kd8) cp_async16(kb + key * KP + c * 16, p.up + kr * p.ldu + (long)h * n.d + c * 8, in);
      else if (c < kd8 + kr8) cp_async16(kb + key * KP + c * 16, p.lat + kr * p.W + n.rot0 + (c - kd8) * 8, in);
      else cp_async16(vb + key * VP + (c - kd8 - kr8) * 16, p.up + kr * p.ldu + (long)n.H * n.d + (long)h * n.dv + (c - kd8 - kr8) * 8, in);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  issue(0, 0);
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-FLT_MAX, -FLT_MAX}, l_run[2] = {0.f, 0.f};
  const int w_last = p.pos[first + min(count, warp * 16 + 16) - 1];       // last key any row of this warp sees (unused when the warp is empty)
  const bool w_live = warp * 16 < count;
  for (int kt = 0; kt < nkt; ++kt) {
    if (kt + 1 < nkt) {
      issue(kt + 1, (kt + 1) & 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    if (w_live && key0 + kt * 64 <= w_last) {
      const uint32_t kb = sbase + (kt & 1) * STAGE, vb = kb + 64 * KP;
      float sacc[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) sacc[i][0] = sacc[i][1] = sacc[i][2] = sacc[i][3] = 0.f;
      const int mi = lane >> 3, rr = lane & 7;
#pragma unroll
      for (int kk = 0; kk < DQ / 16; ++kk)
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          uint32_t b0, b1, b2, b3;
          lp_ldsm_x4(kb + (np * 16 + (mi >> 1) * 8 + rr) * KP + kk * 32 + (mi & 1) * 16, b0, b1, b2, b3);
          lp_mma(sacc[2 * np], qf[kk], b0, b1);
          lp_mma(sacc[2 * np + 1], qf[kk], b2, b3);
        }
      float mx[2] = {-FLT_MAX, -FLT_MAX};
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int dist = r_pos[e >> 1] - (key0 + kt * 64 + nt * 8 + 2 * t + (e & 1));
          const float v = (unsigned)dist < (unsigned)win ? sacc[nt][e] * p.scale_log2 : -FLT_MAX;
          sacc[nt][e] = v;
          mx[e >> 1] = fmaxf(mx[e >> 1], v);
        }
      float corr[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
        mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
        const float mn = fmaxf(m_run[e], mx[e]);
        corr[e] = m_run[e] == -FLT_MAX ? 0.f : exp2f(m_run[e] - mn);
        m_run[e] = mn;
        l_run[e] *= corr[e];
      }
      uint32_t ph[4][4], pl[4][4];          // weights as A fragments: leading bf16 term and the remainder
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        float pv[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          pv[e] = sacc[nt][e] == -FLT_MAX ? 0.f : exp2f(sacc[nt][e] - m_run[e >> 1]);
          l_run[e >> 1] += pv[e];
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const uint32_t hi = lp_pack(pv[2 * e], pv[2 * e + 1]);
          ph[nt >> 1][(nt & 1) * 2 + e] = hi;
          pl[nt >> 1][(nt & 1) * 2 + e] = lp_pack(pv[2 * e] - __uint_as_float(hi << 16), pv[2 * e + 1] - __uint_as_float(hi & 0xffff0000u));
        }
      }
#pragma unroll
      for (int i = 0; i < DV / 8; ++i) {
        o[i][0] *= corr[0];
        o[i][1] *= corr[0];
        o[i][2] *= corr[1];
        o[i][3] *= corr[1];
      }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks)
#pragma unroll
        for (int dp = 0; dp < DV / 16; ++dp) {
          uint32_t b0, b1, b2, b3;
          lp_ldsm_x4_t(vb + (ks * 16 + (mi & 1) * 8 + rr) * VP + dp * 32 + (mi >> 1) * 16, b0, b1, b2, b3);
          lp_mma(o[2 * dp], ph[ks], b0, b1);
          lp_mma(o[2 * dp + 1], ph[ks], b2, b3);
          lp_mma(o[2 * dp], pl[ks], b0, b1);
          lp_mma(o[2 * dp + 1], pl[ks], b2, b3);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 1);
    l_run[e] += __shfl_xor_sync(0xffffffffu, l_run[e], 2);
    if (!r_ok[e]) continue;
    const float inv = 1.f / l_run[e];
    __nv_bfloat16* orow = p.out + (long)r_row[e] * p.ldo + (long)h * n.dv;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
      if (i * 8 < n.dv) *reinterpret_cast<uint32_t*>(orow + i * 8 + 2 * t) = lp_pack(o[i][2 * e] * inv, o[i][2 * e + 1] * inv);
  }
}

template <int DQ, int DV>
static int launch_latent_prefill(const LatentPrefill& p, int ntiles, cudaStream_t st) {
  constexpr int smem = 2 * 64 * (DQ * 2 + 16 + DV * 2 + 16);
  static_assert(smem <= 227 * 1024, "shared memory budget");
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(latent_prefill_kernel<DQ, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  launch_pdl(latent_prefill_kernel<DQ, DV>, dim3(ntiles, p.n.H), dim3(128), smem, st, p);
  return (int)cudaGetLastError();
}

}  // namespace ve
#include "latent_tc.cuh"

using namespace ve;

#define VE_LDIMS int H, int d, int rot, int dv, int kr, int rot0, int W, int pitch
#define VE_LMAKE LatentDims{H, d, rot, dv, kr, rot0, W, pitch}
static bool ldims_ok(const LatentDims& n) {
  return n.H > 0 && n.d > 0 && n.rot >= 0 && n.rot % 2 == 0 && n.rot <= 256 && n.dv > 0 && n.kr > 0 && n.rot0 >= n.kr && n.W >= n.rot0 + n.rot && n.pitch >= n.W;
}

extern "C" {

// x32, kv32: q, kv rows are fp32 (else bf16); f32: q, kv, q_out, pool fp32 (else bf16). q_out null: only the cache row is written.
int ve_latent_rope_store(VE_LDIMS, const void* q, long ldq, void* qo, long ldqo, const void* kv, long ldkv, int x32, int kv32, const void* w,
                         const void* freq, float mul, const void* pos, const void* slot, const void* page_table, int max_pages, void* pool, int rows, float eps, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const LatentDims n = VE_LMAKE;
  if (!ldims_ok(n)) return cudaErrorInvalidValue;
  const LatentTurn tn{(const double*)freq, mul};
#define VE_RS(X, K, T) launch_pdl(latent_rope_store_kernel<X, K, T>, dim3(rows), dim3(256), 0, st, n, (const X*)q, ldq, (T*)qo, ldqo, (const K*)kv, ldkv, \
    (const float*)w, tn, (const int*)pos, (const int*)slot, (const int*)page_table, max_pages, (T*)pool, eps)
  if (f32) VE_RS(float, float, float);
  else if (x32) VE_RS(float, float, __nv_bfloat16);
  else if (kv32) VE_RS(__nv_bfloat16, float, __nv_bfloat16);
  else VE_RS(__nv_bfloat16, __nv_bfloat16, __nv_bfloat16);
#undef VE_RS
  VE_CHECK_LAUNCH();
}

// q_abs [rows][H][qw] (qw >= rot0 + rot; columns outside the latent and the rotated part are written as zero).
int ve_latent_absorb(VE_LDIMS, const void* q, long ldq, const void* kv, long ldkv, int x32, int kv32, const void* w, const void* w_uk,
                     const void* freq, float mul, const void* pos, const void* slot, const void* page_table, int max_pages, void* pool, void* q_abs, int qw, int rows, float eps,
                     int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const LatentDims n = VE_LMAKE;
  if (!ldims_ok(n) || qw < rot0 + rot) return cudaErrorInvalidValue;
  const bool al = !((uintptr_t)w_uk & 15);
  const LatentTurn tn{(const double*)freq, mul};
#define VE_AB(V, X, K, T) launch_pdl(latent_absorb_kernel<V, X, K, T>, dim3(rows, H + 1, (kr + 8 * V - 1) / (8 * V)), dim3(128), 0, st, n, (const X*)q, ldq, \
    (const K*)kv, ldkv, (const float*)w, (const T*)w_uk, tn, (const int*)pos, (const int*)slot, (const int*)page_table, max_pages, (T*)pool, (T*)q_abs, qw, eps)
#define VE_AB_V(V, X, K, T) do { if (al && kr % V == 0) VE_AB(V, X, K, T); else VE_AB(1, X, K, T); } while (0)
  if (f32) VE_AB_V(4, float, float, float);
  else if (x32) VE_AB_V(8, float, float, __nv_bfloat16);
  else if (kv32) VE_AB_V(8, __nv_bfloat16, float, __nv_bfloat16);
  else VE_AB_V(8, __nv_bfloat16, __nv_bfloat16, __nv_bfloat16);
#undef VE_AB_V
#undef VE_AB
  VE_CHECK_LAUNCH();
}

int ve_latent_attn(VE_LDIMS, const void* q_abs, int qw, const void* pos, const void* slot, const void* page_table, int max_pages, const void* pool,
                   float scale, int window, void* o_lat, int rows, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const LatentDims n = VE_LMAKE;
  if (!ldims_ok(n) || kr > 1024 || qw > 4096) return cudaErrorInvalidValue;
#define VE_LA(NC, T) launch_pdl(latent_attn_kernel<NC, T>, dim3(rows, H), dim3(128), (size_t)(qw + 4 * NC * 32) * 4, st, n, (const T*)q_abs, qw, (const int*)pos, \
    (const int*)slot, (const int*)page_table, max_pages, (const T*)pool, scale, window > 0 ? window : INT_MAX, (float*)o_lat)
#define VE_LA_T(T) do { if (kr <= 128) VE_LA(4, T); else if (kr <= 256) VE_LA(8, T); else if (kr <= 512) VE_LA(16, T); else VE_LA(32, T); } while (0)
  if (f32) VE_LA_T(float);
  else VE_LA_T(__nv_bfloat16);
#undef VE_LA_T
#undef VE_LA
  VE_CHECK_LAUNCH();
}

int ve_latent_expand(VE_LDIMS, const void* o_part, const void* lse, int nsplit, int ldp, const void* w_uv, const void* slot, void* out, long ldo, int rows,
                     int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  const LatentDims n = VE_LMAKE;
  if (!ldims_ok(n) || nsplit < 1 || nsplit > 64 || kr > 3072) return cudaErrorInvalidValue;
  const bool al = !((uintptr_t)w_uv & 15);
  const int vper = rows * H >= 296 ? dv : rows * H >= 74 ? 32 : 16;
#define VE_EX(V, T) launch_pdl(latent_expand_kernel<V, T>, dim3(rows, H, (dv + vper - 1) / vper), dim3(512), (size_t)kr * 16, st, n, (const float*)o_part, \
    (const float*)lse, nsplit, ldp, (const T*)w_uv, (const int*)slot, (T*)out, ldo, vper)
  if (f32) {
    if (al && kr % 4 == 0) VE_EX(4, float);
    else VE_EX(1, float);
  } else {
    if (al && kr % 8 == 0) VE_EX(8, __nv_bfloat16);
    else VE_EX(1, __nv_bfloat16);
  }
#undef VE_EX
  VE_CHECK_LAUNCH();
}

// seg_base [nseg]: first output row of every sequence (ascending); rows [seg_base[g], seg_base[g + 1]) are its positions seg_start[g], + 1, ...
int ve_latent_gather(const void* pool, int pitch, const void* page_table, int max_pages, const void* seg_slot, const void* seg_base, const void* seg_start,
                     int nseg, void* out, int W, int total, cudaStream_t st) {
  if (total <= 0) return 0;
  if (W % 8 || pitch % 8 || W > pitch || nseg < 1) return cudaErrorInvalidValue;
  const long items = (long)total * (W / 8);
  const long blocks = (items + 255) / 256;
  launch_pdl(latent_gather_kernel, dim3((unsigned)(blocks < 148 * 8 ? blocks : 148 * 8)), dim3(256), 0, st, (const __nv_bfloat16*)pool, pitch,
             (const int*)page_table, max_pages, (const int*)seg_slot, (const int*)seg_base, (const int*)seg_start, nseg, (__nv_bfloat16*)out, W, total);
  VE_CHECK_LAUNCH();
}

// Widths d, rot and dv multiples of 8, d + rot <= 256, dv <= 256; all bases and pitches 16-byte aligned (bf16).
int ve_latent_prefill(VE_LDIMS, const void* q, long ldq, const void* up, long ldu, const void* lat, int lat_w, const void* pos, const void* tile_first,
                      const void* tile_count, const void* tile_base, const void* tile_key0, int ntiles, int window, void* out, long ldo, float scale,
                      cudaStream_t st) {
  if (ntiles <= 0) return 0;
  const LatentDims n = VE_LMAKE;
  if (!ldims_ok(n) || d % 8 || rot % 8 || dv % 8 || rot0 % 8 || lat_w % 8 || ldq % 8 || ldu % 8 || ldo % 2 || d + rot > 256 || dv > 256 ||
      ((uintptr_t)up & 15) || ((uintptr_t)lat & 15) || ((uintptr_t)q & 3) || ((uintptr_t)out & 3)) return cudaErrorInvalidValue;
  LatentPrefill p{n, (const __nv_bfloat16*)q, ldq, (const __nv_bfloat16*)up, ldu, (const __nv_bfloat16*)lat, lat_w, (const int*)pos, (const int*)tile_first,
                  (const int*)tile_count, (const int*)tile_base, (const int*)tile_key0, window > 0 ? window : INT_MAX, (__nv_bfloat16*)out, ldo,
                  scale * 1.4426950408889634f};
  const int q_w = d + rot;
  if (dv <= 64) {
    if (q_w <= 64) return launch_latent_prefill<64, 64>(p, ntiles, st);
    if (q_w <= 128) return launch_latent_prefill<128, 64>(p, ntiles, st);
    return launch_latent_prefill<256, 64>(p, ntiles, st);
  }
  if (dv <= 128) {
    if (q_w <= 128) return launch_latent_prefill<128, 128>(p, ntiles, st);
    if (q_w <= 192) return launch_latent_prefill<192, 128>(p, ntiles, st);
    return launch_latent_prefill<256, 128>(p, ntiles, st);
  }
  return launch_latent_prefill<256, 256>(p, ntiles, st);
}

// The same on tcgen05: tiles of at most 128 rows; d and rot in at most three chunks of 64 columns together, dv <= 128. up
// [up_rows][...] and lat [up_rows][lat_w] are read through tensor maps.
int ve_latent_prefill_tc(VE_LDIMS, const void* q, long ldq, const void* up, long ldu, const void* lat, int lat_w, long up_rows, const void* pos,
                         const void* tile_first, const void* tile_count, const void* tile_base, const void* tile_key0, int ntiles, int window, void* out,
                         long ldo, float scale, void* status, cudaStream_t st) {
  if (ntiles <= 0) return 0;
  const LatentDims n = VE_LMAKE;
  const int uc = (d + 63) / 64, qc = uc + (rot + 63) / 64, vc = (dv + 63) / 64;
  if (!ldims_ok(n) || d % 8 || rot % 8 || dv % 8 || rot0 % 8 || lat_w % 8 || ldq % 8 || ldu % 8 || ldo % 8 || qc > 3 || vc > 2 || scale <= 0.f ||
      ((uintptr_t)q & 15) || ((uintptr_t)out & 15)) return cudaErrorInvalidValue;
  CUtensorMap um, rm;
  int rc = make_tmap_2d(&um, up, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, up_rows, (uint64_t)H * (d + dv), (uint64_t)ldu * 2, 64, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  rc = make_tmap_2d(&rm, lat, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, up_rows, lat_w, (uint64_t)lat_w * 2, 64, 64, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  LatentTc p{n, (const __nv_bfloat16*)q, ldq, (const int*)pos, (const int*)tile_first, (const int*)tile_count, (const int*)tile_base,
             (const int*)tile_key0, window > 0 ? window : INT_MAX, (__nv_bfloat16*)out, ldo, scale * 1.4426950408889634f, uc, (int*)status};
  if (vc == 1) {
    if (qc == 1) return launch_latent_tc<1, 1>(p, um, rm, ntiles, st);
    if (qc == 2) return launch_latent_tc<2, 1>(p, um, rm, ntiles, st);
    return launch_latent_tc<3, 1>(p, um, rm, ntiles, st);
  }
  if (qc == 1) return launch_latent_tc<1, 2>(p, um, rm, ntiles, st);
  if (qc == 2) return launch_latent_tc<2, 2>(p, um, rm, ntiles, st);
  return launch_latent_tc<3, 2>(p, um, rm, ntiles, st);
}

}  // extern "C"
