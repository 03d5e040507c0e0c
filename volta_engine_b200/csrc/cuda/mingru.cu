// Gated recurrence per channel whose gate and candidate read the current row alone (minGRU): one fp32 state S [width] per slot with
//     S_t = (1 - z_t) S_(t-1) + z_t c_t,      y_t = S_t silu(g_t)
// over fp32 projection rows [ gate z (width) | candidate u (width) | output gate g (width) ]; z = sigmoid, c = u + 1/2 for u >= 0 and
// sigmoid(u) below. A step is an affine map of the state, and so is any run of rows: S -> A S + B with A between zero and one.
//   mingru_step    walks the rows of a segment in order (decode rows, short portions); a thread per channel
//   mingru_chunk   prompt portions, chunks of up to 128 rows in four parts: (a) the maps of all parts and chunks at once, (b) every part
//                  starts from its segment's state through the maps in front of it and walks its rows
// A segment whose first row is at position 0 starts from a zero state. Everything is fp32; no fast-math in this file.
#include "rowmath.cuh"
#include "slot_rows.cuh"

namespace ve {

constexpr int kGruCols = 64, kGruParts = 4, kGruAhead = 8;

struct GruRows {
  const float* proj; long ld;
  const int* pos; const int* slot;
  const int* seg_first; const int* seg_count; int rows;
  float* state;                             // [slots][W]
  int W, cols;                              // cols >= W: columns of the output (zero behind the width)
  long ldo;
};

VE_DEVINL float gru_candidate(float u) { return u >= 0.f ? u + 0.5f : sigmoid_of(u); }
// sigmoid(z) and sigmoid(-z) from one exponential that cannot overflow
VE_DEVINL void gru_gates(float z, float& take, float& keep) {
  const float e = expf(-fabsf(z)), r = 1.f / (1.f + e);
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
    out[(long)i * a.ldo + c] = from_f<T>(live ? S * silu_of(g) : 0.f);
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
  float2* total;                            // [chunks][W]: the map (A, B) of a chunk
  float2* part;                             // [chunks][kGruParts][W]: of its parts
  float* start;                             // [segments][W]: the state in front of a segment
  int W, cols;
  long ldo;
};

// grid (columns / 64, chunks), block (64, 4): a thread is a channel of a part.
__global__ void __launch_bounds__(kGruCols * kGruParts) mingru_maps_kernel(const GruChunks a) {
  __shared__ float2 maps[kGruParts][kGruCols];
  grid_dep_wait();
  grid_dep_launch();
  const int c = blockIdx.x * kGruCols + threadIdx.x, y = threadIdx.y, k = blockIdx.y, first = a.chunk_first[k], count = a.chunk_count[k];
  const int seg = a.chunk_seg[k], slot = a.slot[first];
  if (slot < 0) return;
  const bool live = c < a.W;
  const int per = (count + kGruParts - 1) / kGruParts, r0 = y * per, r1 = min(count, r0 + per);
  if (live && y == 0 && k == a.seg_chunk0[seg]) a.start[(long)seg * a.W + c] = a.pos[first] != 0 ? a.state[(long)slot * a.W + c] : 0.f;
  float A = 1.f, B = 0.f;
  const float* row = a.proj + (long)(first + r0) * a.ld + c;
  for (int r = r0; r < r1; r += kGruAhead, row += kGruAhead * a.ld) {
    float z[kGruAhead], u[kGruAhead];
#pragma unroll
    for (int j = 0; j < kGruAhead; ++j) {
      const bool in = live && r + j < r1;
      z[j] = in ? row[j * a.ld] : 0.f;
      u[j] = in ? row[j * a.ld + a.W] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < kGruAhead; ++j)
      if (r + j < r1) {
        float take, keep;
        gru_gates(z[j], take, keep);
        B = fmaf(keep, B, take * gru_candidate(u[j]));
        A *= keep;
      }
  }
  maps[y][threadIdx.x] = make_float2(A, B);
  if (live) a.part[((long)k * kGruParts + y) * a.W + c] = make_float2(A, B);
  __syncthreads();
  if (y || !live) return;
#pragma unroll
  for (int j = 1; j < kGruParts; ++j) {
    const float2 m = maps[j][threadIdx.x];
    B = fmaf(m.x, B, m.y);
    A *= m.x;
  }
  a.total[(long)k * a.W + c] = make_float2(A, B);
}

template <typename T>
__global__ void __launch_bounds__(kGruCols * kGruParts) mingru_out_kernel(const GruChunks a, T* __restrict__ out) {
  grid_dep_wait();
  grid_dep_launch();
  const int c = blockIdx.x * kGruCols + threadIdx.x, y = threadIdx.y, k = blockIdx.y, first = a.chunk_first[k], count = a.chunk_count[k];
  const int seg = a.chunk_seg[k], slot = a.slot[first];
  if (slot < 0 || c >= a.cols) return;
  const bool live = c < a.W;
  const int per = (count + kGruParts - 1) / kGruParts, r0 = y * per, r1 = min(count, r0 + per);
  if (r0 >= r1) return;
  float S = live ? a.start[(long)seg * a.W + c] : 0.f;
  if (live) {
#pragma unroll 8
    for (int j = a.seg_chunk0[seg]; j < k; ++j) {
      const float2 m = a.total[(long)j * a.W + c];
      S = fmaf(m.x, S, m.y);
    }
    for (int j = 0; j < y; ++j) {
      const float2 m = a.part[((long)k * kGruParts + j) * a.W + c];
      S = fmaf(m.x, S, m.y);
    }
  }
  const float* row = a.proj + (long)(first + r0) * a.ld + c;
  for (int r = r0; r < r1; r += kGruAhead, row += kGruAhead * a.ld) {
    float z[kGruAhead], u[kGruAhead], g[kGruAhead];
#pragma unroll
    for (int j = 0; j < kGruAhead; ++j) {
      const bool in = live && r + j < r1;
      z[j] = in ? row[j * a.ld] : 0.f;
      u[j] = in ? row[j * a.ld + a.W] : 0.f;
      g[j] = in ? row[j * a.ld + 2 * a.W] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < kGruAhead; ++j)
      if (r + j < r1) {
        float take, keep;
        gru_gates(z[j], take, keep);
        S = fmaf(keep, S, take * gru_candidate(u[j]));
        out[(long)(first + r + j) * a.ldo + c] = from_f<T>(live ? S * silu_of(g[j]) : 0.f);
      }
  }
  if (live && r1 == count && k == a.seg_chunk0[seg + 1] - 1) a.state[(long)slot * a.W + c] = S;
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

// The chunked form over a table of chunks (a segment's chunks follow each other). total, part, start: scratch (see GruChunks).
int ve_mingru_chunk(const void* proj, long ld, const void* pos, const void* slot, const void* chunk_seg, const void* chunk_first, const void* chunk_count,
                    const void* seg_chunk0, int chunks, void* state, void* total, void* part, void* start, void* out, long ldo, int W, int cols, int f32,
                    cudaStream_t st) {
  if (chunks <= 0) return 0;
  if (W < 1 || cols < W || ldo < cols || ld < 3l * W) return cudaErrorInvalidValue;
  const GruChunks a{(const float*)proj, ld, (const int*)pos, (const int*)slot, (const int*)chunk_seg, (const int*)chunk_first, (const int*)chunk_count,
                    (const int*)seg_chunk0, (float*)state, (float2*)total, (float2*)part, (float*)start, W, cols, ldo};
  const dim3 block(kGruCols, kGruParts);
  launch_pdl(mingru_maps_kernel, dim3((W + kGruCols - 1) / kGruCols, chunks), block, 0, st, a);
  if (f32) launch_pdl(mingru_out_kernel<float>, dim3((cols + kGruCols - 1) / kGruCols, chunks), block, 0, st, a, (float*)out);
  else launch_pdl(mingru_out_kernel<__nv_bfloat16>, dim3((cols + kGruCols - 1) / kGruCols, chunks), block, 0, st, a, (__nv_bfloat16*)out);
  VE_CHECK_LAUNCH();
}

}  // extern "C"
