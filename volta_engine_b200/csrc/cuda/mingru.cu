// Gated recurrence per channel whose gate and candidate read the current row alone (minGRU): one fp32 state S [width] per slot with
//     S_t = (1 - z_t) S_(t-1) + z_t c_t,      y_t = S_t silu(g_t)
// over fp32 projection rows [ gate z (width) | candidate u (width) | output gate g (width) ]; z = sigmoid, c = u + 1/2 for u >= 0 and
// sigmoid(u) below. A step is an affine map of the state, and so is any run of rows: S -> A S + B with A between zero and one.
//   mingru_step    walks the rows of a segment in order (decode rows, short portions); a thread per channel
//   mingru_chunk   prompt portions, chunks of up to 128 rows in 16 parts: (a) the maps of all chunks at once, (b) every part starts from its
//                  segment's state through the maps of the chunks and parts in front of it and walks its rows in registers
// A segment whose first row is at position 0 starts from a zero state. Everything is fp32; no fast-math in this file.
#include "rowmath.cuh"
#include "slot_rows.cuh"

namespace ve {

constexpr int kGruCols = 64;                            // channels of a CTA of the stepped kernel
constexpr int kGruLanes = 32, kGruParts = 16, kGruRows = 8;      // of a CTA of the chunked kernels: a chunk has at most 16 x 8 rows

struct GruRows {
  const float* proj; long ld;
  const int* pos; const int* slot;
  const int* seg_first; const int* seg_count; int rows;
  float* state;                             // [slots][W]
  int W, cols;                              // cols >= W: columns of the output (zero behind the width)
  long ldo;
};

// exp(-|x|) and 1 / (1 + exp(-|x|)): the product with log2(e) is rounded once and its error put back, so the error stays at a few units in
// the last place for any x; the quotient's divisor lies between one and two.
VE_DEVINL void gru_exp(float x, float& e, float& r) {
  const float a = -fabsf(x), y = a * 1.4426950408889634f, d = fmaf(a, 1.4426950408889634f, -y), p = ex2_approx(y);
  e = fmaf(p, 0.6931471805599453f * d, p);
  r = rcp_approx(1.f + e);
}
VE_DEVINL float gru_sigmoid(float x) {
  float e, r;
  gru_exp(x, e, r);
  return x >= 0.f ? r : e * r;
}
VE_DEVINL float gru_candidate(float u) {
  float e, r;
  gru_exp(u, e, r);
  return u >= 0.f ? u + 0.5f : e * r;
}
// sigmoid(z) and sigmoid(-z)
VE_DEVINL void gru_gates(float z, float& take, float& keep) {
  float e, r;
  gru_exp(z, e, r);
  take = z >= 0.f ? r : e * r;
  keep = z >= 0.f ? e * r : r;
}

// grid (columns / 64, segments or rows), 64 threads.
template <typename T>
__global__ void __launch_bounds__(kGruCols) mingru_step_kernel(const GruRows a, T* __restrict__ out) {
  grid_dep_wait();
  grid_dep_launch();
  const int c = blockIdx.x * kGruCols + threadIdx.x;
  int left = 0;
  int i = segment_of(a, blockIdx.y, left);
  if (i < 0) {
    if (!a.seg_first && a.slot[blockIdx.y] < 0 && c < a.cols) out[blockIdx.y * a.ldo + c] = from_f<T>(0.f);      // a row that stands for nothing
    return;
  }
  const int s = a.slot[i];
  if (s < 0 || c >= a.cols) return;
  const bool live = c < a.W;
  float* st = a.state + (long)s * a.W + c;
  float S = live && a.pos[i] != 0 ? *st : 0.f;
  const float* row = a.proj + (long)i * a.ld + c;
  float z = 0.f, u = 0.f, g = 0.f;
  if (live) {
    z = row[0];
    u = row[a.W];
    g = row[2 * a.W];
  }
  while (i >= 0) {
    const int nxt = next_row(a, i, left);
    --left;
    float z1 = 0.f, u1 = 0.f, g1 = 0.f;
    if (nxt >= 0 && live) {
      row = a.proj + (long)nxt * a.ld + c;
      z1 = row[0];
      u1 = row[a.W];
      g1 = row[2 * a.W];
    }
    float take, keep;
    gru_gates(z, take, keep);
    S = fmaf(keep, S, take * gru_candidate(u));
    out[(long)i * a.ldo + c] = from_f<T>(live ? S * (g * gru_sigmoid(g)) : 0.f);
    z = z1;
    u = u1;
    g = g1;
    i = nxt;
  }
  if (live) *st = S;
}

struct GruChunks {
  const float* proj; long ld;
  const int* pos; const int* slot;
  const int* chunk_seg; const int* chunk_first; const int* chunk_count; const int* seg_chunk0;
  float* state;
  float* total;                             // [chunks][2][W]: the map (A, B) of a chunk
  float* start;                             // [segments][W]: the state in front of a segment
  int W, cols;
  long ldo;
};

// V columns of a row (V 2: all pitches, bases and widths are multiples of two elements).
template <int V> struct GruVec { float v[V]; };
template <int V> VE_DEVINL GruVec<V> gru_load(const float* p) {
  GruVec<V> x;
  if (V == 2) {
    const float2 t = *reinterpret_cast<const float2*>(p);
    x.v[0] = t.x;
    x.v[V - 1] = t.y;
  } else x.v[0] = *p;
  return x;
}
template <int V> VE_DEVINL void gru_store(float* p, const GruVec<V>& x) {
  if (V == 2) *reinterpret_cast<float2*>(p) = make_float2(x.v[0], x.v[V - 1]);
  else *p = x.v[0];
}
template <int V> VE_DEVINL void gru_store(__nv_bfloat16* p, const GruVec<V>& x) {
  if (V == 2) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(x.v[0], x.v[V - 1]);
  else *p = f2bf(x.v[0]);
}

// A thread is V channels of a part (block (32, 16): a warp per part): its rows' maps stay in registers.
template <int V> struct GruPart {
  GruVec<V> keep[kGruRows], add[kGruRows];
  float A[V], B[V];
  int n;
  const float* row;                         // first row, first channel

  VE_DEVINL GruPart(const GruChunks& a, int c, int y, int first, int count) {
    const int per = (count + kGruParts - 1) / kGruParts, r0 = y * per;
    n = max(0, min(count, r0 + per) - r0);
    row = a.proj + (long)(first + (n ? r0 : 0)) * a.ld + c;
    const bool live = c < a.W;
    GruVec<V> z[kGruRows], u[kGruRows];
#pragma unroll
    for (int r = 0; r < kGruRows; ++r) {
      const bool in = live && r < n;
#pragma unroll
      for (int e = 0; e < V; ++e) z[r].v[e] = u[r].v[e] = 0.f;
      if (in) {
        z[r] = gru_load<V>(row + r * a.ld);
        u[r] = gru_load<V>(row + r * a.ld + a.W);
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      A[e] = 1.f;
      B[e] = 0.f;
#pragma unroll
      for (int r = 0; r < kGruRows; ++r)
        if (r < n) {
          float take, k;
          gru_gates(z[r].v[e], take, k);
          keep[r].v[e] = k;
          add[r].v[e] = take * gru_candidate(u[r].v[e]);
          B[e] = fmaf(k, B[e], add[r].v[e]);
          A[e] *= k;
        }
    }
  }
};

// grid (columns / (32 V), chunks)
template <int V>
__global__ void __launch_bounds__(kGruLanes * kGruParts, 2) mingru_maps_kernel(const GruChunks a) {
  __shared__ float2 maps[kGruParts][kGruLanes * V];
  grid_dep_wait();
  grid_dep_launch();
  const int x = threadIdx.x, y = threadIdx.y, c0 = blockIdx.x * kGruLanes * V, k = blockIdx.y, first = a.chunk_first[k], count = a.chunk_count[k];
  const int seg = a.chunk_seg[k], slot = a.slot[first];
  if (slot < 0) return;
  const GruPart<V> p(a, c0 + x * V, y, first, count);
#pragma unroll
  for (int e = 0; e < V; ++e) maps[y][x * V + e] = make_float2(p.A[e], p.B[e]);
  __syncthreads();
  const int i = y * kGruLanes + x, c = c0 + i;
  if (i >= kGruLanes * V || c >= a.W) return;
  float A = 1.f, B = 0.f;
#pragma unroll
  for (int j = 0; j < kGruParts; ++j) {
    const float2 m = maps[j][i];
    B = fmaf(m.x, B, m.y);
    A *= m.x;
  }
  a.total[2l * k * a.W + c] = A;
  a.total[(2l * k + 1) * a.W + c] = B;
  if (k == a.seg_chunk0[seg]) a.start[(long)seg * a.W + c] = a.pos[first] != 0 ? a.state[(long)slot * a.W + c] : 0.f;
}

template <int V, typename T>
__global__ void __launch_bounds__(kGruLanes * kGruParts, 2) mingru_out_kernel(const GruChunks a, T* __restrict__ out) {
  __shared__ float2 maps[kGruParts][kGruLanes * V];
  grid_dep_wait();
  grid_dep_launch();
  const int x = threadIdx.x, y = threadIdx.y, c = blockIdx.x * kGruLanes * V + x * V, k = blockIdx.y, first = a.chunk_first[k], count = a.chunk_count[k];
  const int seg = a.chunk_seg[k], slot = a.slot[first];
  if (slot < 0) return;
  const GruPart<V> p(a, c, y, first, count);
  const bool live = c < a.W;
#pragma unroll
  for (int e = 0; e < V; ++e) maps[y][x * V + e] = make_float2(p.A[e], p.B[e]);
  GruVec<V> S;
#pragma unroll
  for (int e = 0; e < V; ++e) S.v[e] = 0.f;
  if (live) {
    S = gru_load<V>(a.start + (long)seg * a.W + c);
#pragma unroll 8
    for (int j = a.seg_chunk0[seg]; j < k; ++j) {
      const GruVec<V> A = gru_load<V>(a.total + 2l * j * a.W + c), B = gru_load<V>(a.total + (2l * j + 1) * a.W + c);
#pragma unroll
      for (int e = 0; e < V; ++e) S.v[e] = fmaf(A.v[e], S.v[e], B.v[e]);
    }
  }
  __syncthreads();
  if (c >= a.cols || !p.n) return;
  GruVec<V> g[kGruRows];
#pragma unroll
  for (int r = 0; r < kGruRows; ++r)
    if (live && r < p.n) g[r] = gru_load<V>(p.row + r * a.ld + 2 * a.W);
  for (int j = 0; j < y; ++j)
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float2 m = maps[j][x * V + e];
      S.v[e] = fmaf(m.x, S.v[e], m.y);
    }
  const int r0 = (int)((p.row - a.proj - c) / a.ld);
#pragma unroll
  for (int r = 0; r < kGruRows; ++r)
    if (r < p.n) {
      GruVec<V> o;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        S.v[e] = fmaf(p.keep[r].v[e], S.v[e], p.add[r].v[e]);
        o.v[e] = live ? S.v[e] * (g[r].v[e] * gru_sigmoid(g[r].v[e])) : 0.f;
      }
      gru_store<V>(out + (long)(r0 + r) * a.ldo + c, o);
    }
  const int per = (count + kGruParts - 1) / kGruParts;
  if (live && y * per + p.n == count && k == a.seg_chunk0[seg + 1] - 1) gru_store<V>(a.state + (long)slot * a.W + c, S);
}

template <int V, typename T>
static int launch_gru_chunks(const GruChunks& a, int chunks, T* out, cudaStream_t st) {
  constexpr int per = kGruLanes * V;
  const dim3 block(kGruLanes, kGruParts);
  launch_pdl(mingru_maps_kernel<V>, dim3((a.W + per - 1) / per, chunks), block, 0, st, a);
  launch_pdl(mingru_out_kernel<V, T>, dim3((a.cols + per - 1) / per, chunks), block, 0, st, a, out);
  return (int)cudaGetLastError();
}

}  // namespace ve

using namespace ve;

extern "C" {

// proj fp32 [rows][ld], state fp32 [slots][W]; out [rows][ldo] fp32 when f32, else bf16: cols >= W columns. nseg > 0: segment table; 0: segments
// from the slots of the rows (a few rows only: every CTA scans them).
int ve_mingru_step(const void* proj, long ld, const void* pos, const void* slot, const void* seg_first, const void* seg_count, int nseg, void* state, void* out,
                   long ldo, int rows, int W, int cols, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (W < 1 || cols < W || ldo < cols || ld < 3l * W) return cudaErrorInvalidValue;
  const GruRows a{(const float*)proj, ld, (const int*)pos, (const int*)slot, nseg > 0 ? (const int*)seg_first : nullptr, (const int*)seg_count, rows, (float*)state,
                  W, cols, ldo};
  const dim3 grid((cols + kGruCols - 1) / kGruCols, nseg > 0 ? nseg : rows);
  if (f32) launch_pdl(mingru_step_kernel<float>, grid, dim3(kGruCols), 0, st, a, (float*)out);
  else launch_pdl(mingru_step_kernel<__nv_bfloat16>, grid, dim3(kGruCols), 0, st, a, (__nv_bfloat16*)out);
  VE_CHECK_LAUNCH();
}

// The chunked form over a table of chunks (at most 128 rows each; a segment's chunks follow each other). total, start: scratch (see GruChunks).
int ve_mingru_chunk(const void* proj, long ld, const void* pos, const void* slot, const void* chunk_seg, const void* chunk_first, const void* chunk_count,
                    const void* seg_chunk0, int chunks, void* state, void* total, void* start, void* out, long ldo, int W, int cols, int f32, cudaStream_t st) {
  if (chunks <= 0) return 0;
  if (W < 1 || cols < W || ldo < cols || ld < 3l * W) return cudaErrorInvalidValue;
  const GruChunks a{(const float*)proj, ld, (const int*)pos, (const int*)slot, (const int*)chunk_seg, (const int*)chunk_first, (const int*)chunk_count,
                    (const int*)seg_chunk0, (float*)state, (float*)total, (float*)start, W, cols, ldo};
  const bool vec = !((W | cols | ld | ldo) & 1) && !(((uintptr_t)proj | (uintptr_t)state | (uintptr_t)total | (uintptr_t)start | (uintptr_t)out) & 7);
  if (f32) return vec ? launch_gru_chunks<2>(a, chunks, (float*)out, st) : launch_gru_chunks<1>(a, chunks, (float*)out, st);
  return vec ? launch_gru_chunks<2>(a, chunks, (__nv_bfloat16*)out, st) : launch_gru_chunks<1>(a, chunks, (__nv_bfloat16*)out, st);
}

}  // extern "C"
