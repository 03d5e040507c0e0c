// Linear attention with a decayed outer-product state, one fp32 state S [dk][dv] per (slot, head):
//     S_t = diag(d_t) S_(t-1) + k_t v_t^T,      o_t = S_t^T q_t
// Two ways to get decay and key from a projection row [ q (H dk) | x (H dk) | v (H dv) | ... ]:
//   MODE 0  constant decay per head (table), k = silu(x), v = silu(v)                     ("lightning" attention)
//   MODE 1  forget gate per channel: f = lower + (1 - lower) sigmoid(x + bias), d = f, k = 1 - f, v as projected   (HGRN2)
// q = silu(q) in both. Gates, decays, states and outputs are fp32; the file is compiled without fast-math.
//
//   linattn_step    walks the rows of a segment in order with the state in registers (decode rows, short portions, and the
//                   all-32-bit form). One CTA per (head, 32 value columns, segment).
//   linattn_chunk_* prompt portions: chunks of 64 rows in parallel. (a) every chunk's own contribution to the state, (b) a scan
//                   over the chunks that turns contributions into start states, (c) outputs from the start state plus the
//                   products inside the chunk. Products run on the tensor cores with both operands split into two bf16
//                   terms where they are not bf16 already (error about 2^-17), so scores and states keep 32-bit quality.
//
// A segment whose first row is at position 0 starts from a zero state. Segments come from a host table (first row, row count)
// or, without one, from the slots of the rows themselves (rows of one slot are consecutive positions in order).
#include "rowmath.cuh"

namespace ve {

struct LinArgs {
  const void* proj; long ld;
  const int* pos; const int* slot;
  const int* seg_first; const int* seg_count;   // null: one CTA row per batch row, the first row of a slot takes them all
  float* state;                                 // [slots][H][dk][dv]
  const float* bias; const float* lower;        // MODE 1: [H dk] each
  const float* decay;                           // MODE 0: [H]
  float* o; long ldo;                           // [rows][H dv]
  int rows, H, dk, dv;
};

// Rows of the segment that blockIdx.z stands for; -1 when there is nothing to do.
VE_DEVINL int segment_of(const LinArgs& a, int z, int& count) {
  if (a.seg_first) {
    count = a.seg_count[z];
    return count > 0 ? a.seg_first[z] : -1;
  }
  const int s = a.slot[z];
  if (s < 0) return -1;
  for (int i = 0; i < z; ++i)
    if (a.slot[i] == s) return -1;
  count = -1;                                   // rows of the slot are found while walking
  return z;
}
VE_DEVINL int next_row(const LinArgs& a, int i, int left) {
  if (a.seg_first) return left > 1 ? i + 1 : -1;
  const int s = a.slot[i];
  for (int j = i + 1; j < a.rows; ++j)
    if (a.slot[j] == s) return j;
  return -1;
}

// block (32, 8): lane = value column, y = key group (channels y, y + 8, ...); NK channels per thread.
template <int NK, typename X, int MODE>
__global__ void __launch_bounds__(256) linattn_step_kernel(const LinArgs a) {
  __shared__ float sq[2][NK * 8], sk[2][NK * 8], sd[2][MODE ? NK * 8 : 8], red[2][8][32];
  const int lane = threadIdx.x, g = threadIdx.y, tid = g * 32 + lane;
  const int h = blockIdx.x, col = blockIdx.y * 32 + lane;
  const bool live = col < a.dv;
  grid_dep_wait();
  grid_dep_launch();
  int left = 0;
  int i = segment_of(a, blockIdx.z, left);
  if (i < 0) return;
  const int s = a.slot[i];
  if (s < 0) return;
  const bool fresh = a.pos[i] == 0;
  float* st = a.state + (((long)s * a.H + h) * a.dk) * a.dv + col;
  float S[NK];
#pragma unroll
  for (int j = 0; j < NK; ++j) {
    const int k = j * 8 + g;
    S[j] = (!fresh && live && k < a.dk) ? st[(long)k * a.dv] : 0.f;
  }
  const float head_decay = MODE == 0 ? a.decay[h] : 0.f;
  float bias = 0.f, low = 0.f;
  if (MODE == 1 && tid < a.dk) {
    bias = a.bias[h * a.dk + tid];
    low = a.lower[h * a.dk + tid];
  }
  const X* base = reinterpret_cast<const X*>(a.proj);
  const long oq = (long)h * a.dk + tid, okx = (long)(a.H + h) * a.dk + tid, ov = (long)2 * a.H * a.dk + (long)h * a.dv + col;
  float rq = 0.f, rx = 0.f, rv = 0.f;
  if (tid < a.dk) {
    rq = to_f(base[i * a.ld + oq]);
    rx = to_f(base[i * a.ld + okx]);
  }
  if (live) rv = to_f(base[i * a.ld + ov]);
  int b = 0, prev = -1;
  while (i >= 0) {
    if (tid < NK * 8) {
      const bool in = tid < a.dk;
      sq[b][tid] = in ? silu_of(rq) : 0.f;
      if (MODE == 0) sk[b][tid] = in ? silu_of(rx) : 0.f;
      else {
        const float z = rx + bias;
        sd[b][tid] = in ? fmaf(1.f - low, sigmoid_of(z), low) : 0.f;
        sk[b][tid] = in ? (1.f - low) * sigmoid_of(-z) : 0.f;
      }
    }
    const float v = MODE == 0 ? silu_of(rv) : rv;
    const int nxt = next_row(a, i, left);
    --left;
    if (nxt >= 0) {
      if (tid < a.dk) {
        rq = to_f(base[nxt * a.ld + oq]);
        rx = to_f(base[nxt * a.ld + okx]);
      }
      if (live) rv = to_f(base[nxt * a.ld + ov]);
    }
    __syncthreads();
    if (prev >= 0 && g == (b << 2) && live) {     // the row in front: its partial sums are complete
      float t = 0.f;
#pragma unroll
      for (int y = 0; y < 8; ++y) t += red[b ^ 1][y][lane];
      a.o[prev * a.ldo + (long)h * a.dv + col] = t;
    }
    float acc = 0.f;
#pragma unroll
    for (int j = 0; j < NK; ++j) {
      const int k = j * 8 + g;
      S[j] = fmaf(S[j], MODE == 0 ? head_decay : sd[b][k], sk[b][k] * v);
      acc = fmaf(S[j], sq[b][k], acc);
    }
    red[b][g][lane] = acc;
    prev = i;
    i = nxt;
    b ^= 1;
  }
  __syncthreads();
  if (g == 0 && live) {
    float t = 0.f;
#pragma unroll
    for (int y = 0; y < 8; ++y) t += red[b ^ 1][y][lane];
    a.o[prev * a.ldo + (long)h * a.dv + col] = t;
  }
#pragma unroll
  for (int j = 0; j < NK; ++j) {
    const int k = j * 8 + g;
    if (live && k < a.dk) st[(long)k * a.dv] = S[j];
  }
}

}  // namespace ve

using namespace ve;

extern "C" {

// mode 0 / 1 as above (bias / lower or decay accordingly). x32: the projection rows are fp32 (else bf16). nseg > 0: segment
// table; 0: segments from the slots of the rows (a few rows only: every CTA scans them).
int ve_linattn_step(const void* proj, long ld, int x32, const void* pos, const void* slot, const void* seg_first, const void* seg_count, int nseg,
                    void* state, const void* bias, const void* lower, const void* decay, void* o, long ldo, int rows, int H, int dk, int dv,
                    int mode, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (dk < 1 || dk > 256 || dv < 1 || H < 1 || (mode == 0 ? !decay : (!bias || !lower))) return cudaErrorInvalidValue;
  LinArgs a{proj, ld, (const int*)pos, (const int*)slot, nseg > 0 ? (const int*)seg_first : nullptr, (const int*)seg_count, (float*)state,
            (const float*)bias, (const float*)lower, (const float*)decay, (float*)o, ldo, rows, H, dk, dv};
  const dim3 grid(H, (dv + 31) / 32, nseg > 0 ? nseg : rows), block(32, 8);
#define VE_LS(NK, X, MODE) launch_pdl(linattn_step_kernel<NK, X, MODE>, grid, block, 0, st, a)
#define VE_LS_M(NK, X) do { if (mode == 0) VE_LS(NK, X, 0); else VE_LS(NK, X, 1); } while (0)
#define VE_LS_X(NK) do { if (x32) VE_LS_M(NK, float); else VE_LS_M(NK, __nv_bfloat16); } while (0)
  if (dk <= 32) VE_LS_X(4);
  else if (dk <= 64) VE_LS_X(8);
  else if (dk <= 128) VE_LS_X(16);
  else VE_LS_X(32);
#undef VE_LS_X
#undef VE_LS_M
#undef VE_LS
  VE_CHECK_LAUNCH();
}

}  // extern "C"
