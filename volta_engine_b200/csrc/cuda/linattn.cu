// Linear attention with a decayed outer-product state, one fp32 state S [dk][dv] per (slot, head):
//     S_t = diag(d_t) S_(t-1) + k_t v_t^T,      o_t = S_t^T q_t
// Three ways to get decay and key from a projection row [ q (H dk) | x (H dk) | v (H dv) | ... ]:
//   MODE 0  constant decay per head (table), k = silu(x), v = silu(v)                     ("lightning" attention), or with `plain` k = x,
//           v as projected, q scaled by a constant                                        (retention)
//   MODE 1  forget gate per channel: f = lower + (1 - lower) sigmoid(x + bias), d = f, k = 1 - f, v as projected   (HGRN2)
//   MODE 2  decay per channel sigmoid(z)^(1 / tau) with z = W a + bias for a low-rank row a of the projection; k = x, v as projected,
//           q scaled by a constant                                                        (gated linear attention)
// q = silu(q) in modes 0 (but for `plain`) and 1. Gates, decays, states and outputs are fp32; the file is compiled without fast-math.
//
//   linattn_decay   the decays of mode 2 as rows (for the chunks; the stepped kernel forms its own)
//   linattn_step    walks the rows of a segment in order with the state in registers (decode rows, short portions, and the
//                   all-32-bit form). One CTA per (head, 32 value columns, segment).
//   linattn_chunk   prompt portions, chunks of up to 128 rows in parallel: (a) every chunk's own contribution to the state,
//                   (b) a scan over the chunks that turns contributions into start states, (c) outputs. A chunk is walked in
//                   blocks of 16 rows with the state in MMA accumulators: held as S^T [dv][dk] its accumulator layout is the
//                   B-operand layout of o = (q prefix) S, so it feeds the tensor cores without leaving the registers.
//                   Decays enter as running products inside a block (never above one, no logarithms, no quotients), the
//                   16 x 16 products of a block itself are formed in fp32 on the CUDA cores. Operands that are not bf16 already
//                   (decayed queries and keys, the state, the block's scores) enter as two bf16 terms each, error about
//                   2^-16; values are bf16.
//
// A segment whose first row is at position 0 starts from a zero state. Segments come from a host table (first row, row count)
// or, without one, from the slots of the rows themselves (rows of one slot are consecutive positions in order).
#include "rowmath.cuh"
#include "slot_rows.cuh"

namespace ve {

struct LinArgs {
  const void* proj; long ld;
  const int* pos; const int* slot;
  const int* seg_first; const int* seg_count;   // null: one CTA row per batch row, the first row of a slot takes them all
  float* state;                                 // [slots][H][dk][dv]
  const float* bias; const float* lower;        // MODE 1: [H dk] each; MODE 2: bias
  const float* decay;                           // MODE 0: [H]
  float* o; long ldo;                           // [rows][H dv]
  int rows, H, dk, dv;
  const float* w2; int rank, a_col;             // MODE 2: [H dk][rank], first column of the low-rank part in a projection row
  float inv_tau, q_scale;
  int plain;                                    // MODE 0: operands as projected, q scaled
};

// sigmoid(z)^inv_tau through the logarithm of the sigmoid, which is exact on both sides
VE_DEVINL float root_decay(float z, float inv_tau) { return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau); }

template <typename X>
VE_DEVINL float lowrank_of(const X* __restrict__ a, const float* __restrict__ w, int rank, float z) {
  float z1 = 0.f;
  int r = 0;
  if ((rank & 3) == 0) {
    float z2 = 0.f, z3 = 0.f;
    for (; r < rank; r += 4) {
      const float4 v = *reinterpret_cast<const float4*>(w + r);
      z = fmaf(v.x, to_f(a[r]), z);
      z1 = fmaf(v.y, to_f(a[r + 1]), z1);
      z2 = fmaf(v.z, to_f(a[r + 2]), z2);
      z3 = fmaf(v.w, to_f(a[r + 3]), z3);
    }
    return (z + z1) + (z2 + z3);
  }
  for (; r < rank; ++r) z = fmaf(w[r], to_f(a[r]), z);
  return z;
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
  const bool plain = MODE == 0 && a.plain;
  float bias = 0.f, low = 0.f;
  if (MODE == 1 && tid < a.dk) {
    bias = a.bias[h * a.dk + tid];
    low = a.lower[h * a.dk + tid];
  }
  const X* base = reinterpret_cast<const X*>(a.proj);
  const long oq = (long)h * a.dk + tid, okx = (long)(a.H + h) * a.dk + tid, ov = (long)2 * a.H * a.dk + (long)h * a.dv + col;
  float rq = 0.f, rx = 0.f, rv = 0.f, rz = 0.f;
  const float* w2 = MODE == 2 && tid < a.dk ? a.w2 + ((long)h * a.dk + tid) * a.rank : nullptr;
  if (MODE == 2 && tid < a.dk) bias = a.bias[h * a.dk + tid];
  if (tid < a.dk) {
    rq = to_f(base[i * a.ld + oq]);
    rx = to_f(base[i * a.ld + okx]);
    if (MODE == 2) rz = lowrank_of(base + i * a.ld + a.a_col, w2, a.rank, bias);
  }
  if (live) rv = to_f(base[i * a.ld + ov]);
  int b = 0, prev = -1;
  while (i >= 0) {
    if (tid < NK * 8) {
      const bool in = tid < a.dk;
      sq[b][tid] = in ? (MODE == 2 || plain ? rq * a.q_scale : silu_of(rq)) : 0.f;
      if (MODE == 0) sk[b][tid] = in ? (plain ? rx : silu_of(rx)) : 0.f;
      else if (MODE == 2) {
        sk[b][tid] = in ? rx : 0.f;
        sd[b][tid] = in ? root_decay(rz, a.inv_tau) : 0.f;
      } else {
        const float z = rx + bias;
        sd[b][tid] = in ? fmaf(1.f - low, sigmoid_of(z), low) : 0.f;
        sk[b][tid] = in ? (1.f - low) * sigmoid_of(-z) : 0.f;
      }
    }
    const float v = MODE == 0 && !plain ? silu_of(rv) : rv;
    const int nxt = next_row(a, i, left);
    --left;
    if (nxt >= 0) {
      if (tid < a.dk) {
        rq = to_f(base[nxt * a.ld + oq]);
        rx = to_f(base[nxt * a.ld + okx]);
        if (MODE == 2) rz = lowrank_of(base + nxt * a.ld + a.a_col, w2, a.rank, bias);
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

// ---------------------------------------------------------------------------------------------- chunked form
struct LinChunkArgs {
  const float* proj; long ld;
  const int* pos; const int* slot;
  const int* chunk_seg; const int* chunk_first; const int* chunk_count; const int* seg_chunk0;   // seg_chunk0 [segments + 1]
  float* state;                         // [slots][H][dk][dv]
  float* start;                         // [chunks][H][dk][dv]: contributions, after the scan start states
  float* total;                         // [chunks][H][dk]: product of a chunk's decays
  const float* bias; const float* lower; const float* decay;
  float* o; long ldo;
  int H, dk, dv, vec;                   // vec: 16-byte copies are aligned
  const float* dec;                     // MODE 2: decays [rows][H dk]
  float q_scale;
  int plain;                            // as above
};

VE_DEVINL void la_ldsm_x4(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
VE_DEVINL void la_ldsm_x4_t(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
VE_DEVINL void la_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
VE_DEVINL void la_split2(float x, float y, uint32_t& hi, uint32_t& lo) {      // two values -> leading bf16 pair and remainder pair
  __nv_bfloat162 t = __floats2bfloat162_rn(x, y);
  hi = *reinterpret_cast<uint32_t*>(&t);
  t = __floats2bfloat162_rn(x - __low2float(t), y - __high2float(t));
  lo = *reinterpret_cast<uint32_t*>(&t);
}
VE_DEVINL void la_put(__nv_bfloat16* hi, __nv_bfloat16* lo, int at, float v) {
  const __nv_bfloat16 h = f2bf(v);
  hi[at] = h;
  lo[at] = f2bf(v - bf2f(h));
}

// grid (chunks, H), 128 threads. OUT false: pass (a), true: pass (c). DK, DV: padded widths (32, 64 or 128).
// MODE 2 brings its decays as rows: they are staged beside the projections, and the block's own products read decays, keys and
// queries where they were staged.
template <int DK, int DV, int MODE, bool OUT>
__global__ void __launch_bounds__(128) linattn_chunk_kernel(const LinChunkArgs a) {
  constexpr int KP = DK + 8, VP = DV + 8;                 // bf16 row pitches: 16 bytes past a multiple of 64 (no ldmatrix conflicts)
  constexpr int MT = DV >= 64 ? DV / 64 : 1;              // 16-column tiles of the value width per warp
  constexpr int NT = DK / 8, RAW = 2 * DK + DV + (MODE == 2 ? DK : 0);           // RAW: floats per staged row [q | x | v (| decay)]
  constexpr int CG = DK / 8;                              // channels per thread in the block's own products
  extern __shared__ __align__(16) uint8_t sm[];
  float* raw = reinterpret_cast<float*>(sm);              // [2][16][RAW]
  float* sf = raw + 2 * 16 * RAW;                         // [16][DK] decays
  float* btot = sf + (MODE == 2 ? 0 : 16 * DK);           // [DK]
  __nv_bfloat16* ksh = reinterpret_cast<__nv_bfloat16*>(btot + DK);   // [16][KP] decayed keys, two terms
  __nv_bfloat16* ksl = ksh + 16 * KP;
  __nv_bfloat16* vs = ksl + 16 * KP;                      // [16][VP]
  __nv_bfloat16* qph = vs + 16 * VP;                      // OUT: [16][KP] decayed queries, two terms
  __nv_bfloat16* qpl = qph + 16 * KP;
  __nv_bfloat16* ah = qpl + 16 * KP;                      // OUT: [16][24] block scores, two terms
  __nv_bfloat16* al = ah + 16 * 24;
  float* apart = reinterpret_cast<float*>(al + 16 * 24);  // OUT: [8][16][17]
  float* sk = apart + 8 * 16 * 17;                        // OUT: [16][DK] keys
  float* sq = sk + 16 * DK;                               // OUT: [16][DK] queries
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  grid_dep_wait();
  grid_dep_launch();
  const int c = blockIdx.x, h = blockIdx.y, seg = a.chunk_seg[c];
  const int first = a.chunk_first[c], count = a.chunk_count[c];
  const int c_begin = a.seg_chunk0[seg], c_end = a.seg_chunk0[seg + 1];
  if (!OUT && c == c_end - 1) return;                     // nobody starts from the last chunk's contribution
  const int slot = a.slot[first];
  if (slot < 0) return;
  const bool single = c_end - c_begin == 1;
  const int v0 = warp * MT * 16;
  const bool wlive = v0 < DV;
  float* st = a.state + ((long)slot * a.H + h) * a.dk * a.dv;
  float* cs = a.start + ((long)c * a.H + h) * a.dk * a.dv;
  const long oq = (long)h * a.dk, ox = (long)(a.H + h) * a.dk, ov = (long)2 * a.H * a.dk + (long)h * a.dv;

  auto from = [&](int part, int row, int col) {           // where column col of a staged part lives
    if (MODE == 2 && part == 3) return a.dec + ((long)(first + row) * a.H + h) * a.dk + col;
    return a.proj + (long)(first + row) * a.ld + (part == 0 ? oq : part == 1 ? ox : ov) + col;
  };
  // rows [16 b, 16 b + 16) of the chunk into raw buffer b & 1 (rows and columns that do not exist: zeros)
  auto stage = [&](int b) {
    float* dst = raw + (b & 1) * 16 * RAW;
    if (a.vec) {
      constexpr int Q4 = RAW / 4;
      for (int i = tid; i < 16 * Q4; i += 128) {
        const int r = i / Q4, w = (i % Q4) * 4, row = b * 16 + r;
        const int part = w < DK ? 0 : (w < 2 * DK ? 1 : (w < 2 * DK + DV ? 2 : 3)), col = part == 3 ? w - 2 * DK - DV : w - part * DK;
        const bool in = row < count && col < (part == 2 ? a.dv : a.dk) && (OUT || part != 0);
        const float* src = in ? from(part, row, col) : a.proj;
        const int n = in ? 16 : 0;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + r * RAW + w)), "l"(src), "r"(n) : "memory");
      }
    } else {
      for (int i = tid; i < 16 * RAW; i += 128) {
        const int r = i / RAW, w = i % RAW, row = b * 16 + r;
        const int part = w < DK ? 0 : (w < 2 * DK ? 1 : (w < 2 * DK + DV ? 2 : 3)), col = part == 3 ? w - 2 * DK - DV : w - part * DK;
        const bool in = row < count && col < (part == 2 ? a.dv : a.dk);
        dst[i] = in ? *from(part, row, col) : 0.f;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int nb = (count + 15) / 16;
  stage(0);

  float S[MT][NT][4];                                     // S^T tile: rows v0 + 16 m + {g, g + 8}, columns 8 n + {2t, 2t + 1}
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int v = v0 + m * 16 + g + (e >> 1) * 8, k = n * 8 + 2 * t + (e & 1);
        float x = 0.f;
        if (OUT && wlive && v < a.dv && k < a.dk) {
          if (!single) x = cs[(long)k * a.dv + v];
          else if (a.pos[first] != 0) x = st[(long)k * a.dv + v];
        }
        S[m][n][e] = x;
      }
  const bool ch = tid < a.dk;
  const float head_decay = MODE == 0 ? a.decay[h] : 0.f;
  const bool plain = MODE == 0 && a.plain;
  float bias = 0.f, low = 0.f, prod = 1.f;
  if (MODE == 1 && ch) {
    bias = a.bias[h * a.dk + tid];
    low = a.lower[h * a.dk + tid];
  }
  for (int b = 0; b < nb; ++b) {
    if (b + 1 < nb) {
      stage(b + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* rw = raw + (b & 1) * 16 * RAW;
    const int live = min(16, count - b * 16);
    // ---- gates: thread = channel
    if (tid < DK) {
      float f[16], k[16], run = 1.f;
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const float x = rw[i * RAW + DK + tid];
        const bool in = ch && i < live;                   // rows behind the end: decay one, key zero
        if (MODE == 0) {
          f[i] = in ? head_decay : 1.f;
          k[i] = in ? (plain ? x : silu_of(x)) : 0.f;
        } else if (MODE == 2) {
          f[i] = in ? rw[i * RAW + 2 * DK + DV + tid] : 1.f;
          k[i] = x;                                       // (zero where there is no row or channel)
        } else {
          const float z = x + bias, e = expf(-fabsf(z)), r = 1.f / (1.f + e);       // sigmoid(z) and sigmoid(-z)
          const float p = z >= 0.f ? r : e * r, n = z >= 0.f ? e * r : r;
          f[i] = in ? fmaf(1.f - low, p, low) : 1.f;
          k[i] = in ? (1.f - low) * n : 0.f;
        }
        run *= f[i];
        if (OUT) {
          const float q = MODE == 2 || plain ? rw[i * RAW + tid] * a.q_scale : in ? silu_of(rw[i * RAW + tid]) : 0.f;
          if (MODE != 2) {
            sf[i * DK + tid] = f[i];
            sk[i * DK + tid] = k[i];
            sq[i * DK + tid] = q;
          }
          la_put(qph, qpl, i * KP + tid, q * run);
        }
      }
      btot[tid] = run;
      prod *= run;
      float suf = 1.f;
#pragma unroll
      for (int i = 15; i >= 0; --i) {
        la_put(ksh, ksl, i * KP + tid, k[i] * suf);
        suf *= f[i];
      }
    }
    for (int i = tid; i < 16 * DV; i += 128) {
      const int r = i / DV, v = i % DV;
      const float x = rw[r * RAW + 2 * DK + v];
      vs[r * VP + v] = f2bf(MODE == 0 && !plain ? silu_of(x) : x);
    }
    __syncthreads();
    float o[MT * 2][4];
    const int mi = lane >> 3, rr = lane & 7;
    if (OUT) {
      // ---- the block's own products in fp32: thread = (key row s, CG channels)
      const int s = tid & 15, c0 = (tid >> 4) * CG;
      constexpr int OP = MODE == 2 ? RAW : DK;            // row pitch of the operands
      const float* of = (MODE == 2 ? rw + 2 * DK + DV : sf) + c0;
      const float* ok = (MODE == 2 ? rw + DK : sk) + c0;
      const float* oqs = (MODE == 2 ? rw : sq) + c0;
      float w[CG], acc[16];
#pragma unroll
      for (int j = 0; j < CG; ++j) w[j] = 0.f;
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < CG; j += 4) {
          const float4 f4 = *reinterpret_cast<const float4*>(of + i * OP + j), q4 = *reinterpret_cast<const float4*>(oqs + i * OP + j);
          const float fv[4] = {f4.x, f4.y, f4.z, f4.w}, qv[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            w[j + e] = i == s ? ok[s * OP + j + e] : w[j + e] * fv[e];
            sum = fmaf(qv[e], w[j + e], sum);
          }
        }
        acc[i] = sum;                                     // zero while i < s
      }
#pragma unroll
      for (int i = 0; i < 16; ++i) apart[((tid >> 4) * 16 + i) * 17 + s] = acc[i];
      // ---- o = (decayed q) S
#pragma unroll
      for (int n = 0; n < MT * 2; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
      if (wlive) {
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          uint32_t qa[4], ql[4];
          la_ldsm_x4(smem_u32(qph + ((mi & 1) * 8 + rr) * KP + kk * 16 + (mi >> 1) * 8), qa);
          la_ldsm_x4(smem_u32(qpl + ((mi & 1) * 8 + rr) * KP + kk * 16 + (mi >> 1) * 8), ql);
#pragma unroll
          for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int e = 0; e < 2; ++e) {                 // value columns g / g + 8 of the tile
              uint32_t h0, l0, h1, l1;
              la_split2(S[m][2 * kk][2 * e], S[m][2 * kk][2 * e + 1], h0, l0);
              la_split2(S[m][2 * kk + 1][2 * e], S[m][2 * kk + 1][2 * e + 1], h1, l1);
              la_mma(o[2 * m + e], qa, h0, h1);
              la_mma(o[2 * m + e], qa, l0, l1);
              la_mma(o[2 * m + e], ql, h0, h1);
            }
        }
      }
      __syncthreads();
      for (int i = tid; i < 256; i += 128) {
        float v = 0.f;
#pragma unroll
        for (int y = 0; y < 8; ++y) v += apart[(y * 16 + (i >> 4)) * 17 + (i & 15)];
        la_put(ah, al, (i >> 4) * 24 + (i & 15), MODE == 2 ? v * a.q_scale : v);
      }
      __syncthreads();
      if (wlive) {
        uint32_t pa[4], pl[4];
        la_ldsm_x4(smem_u32(ah + ((mi & 1) * 8 + rr) * 24 + (mi >> 1) * 8), pa);
        la_ldsm_x4(smem_u32(al + ((mi & 1) * 8 + rr) * 24 + (mi >> 1) * 8), pl);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t vb[4];                                 // B operand: rows = keys, columns = values
          la_ldsm_x4_t(smem_u32(vs + ((mi & 1) * 8 + rr) * VP + v0 + m * 16 + (mi >> 1) * 8), vb);
          la_mma(o[2 * m], pa, vb[0], vb[1]);
          la_mma(o[2 * m + 1], pa, vb[2], vb[3]);
          la_mma(o[2 * m], pl, vb[0], vb[1]);
          la_mma(o[2 * m + 1], pl, vb[2], vb[3]);
        }
#pragma unroll
        for (int n = 0; n < MT * 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int row = b * 16 + g + (e >> 1) * 8, v = v0 + n * 8 + 2 * t + (e & 1);
            if (row < count && v < a.dv) a.o[(long)(first + row) * a.ldo + (long)h * a.dv + v] = o[n][e];
          }
      }
    }
    // ---- S^T = S^T diag(block decay) + V^T (decayed k)
    if (wlive) {
      uint32_t va[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)                        // A operand: rows = values, columns = keys (transposed read)
        la_ldsm_x4_t(smem_u32(vs + ((mi >> 1) * 8 + rr) * VP + v0 + m * 16 + (mi & 1) * 8), va[m]);
#pragma unroll
      for (int n2 = 0; n2 < NT / 2; ++n2) {
        uint32_t kh[4], kl[4];
        la_ldsm_x4_t(smem_u32(ksh + ((mi & 1) * 8 + rr) * KP + n2 * 16 + (mi >> 1) * 8), kh);
        la_ldsm_x4_t(smem_u32(ksl + ((mi & 1) * 8 + rr) * KP + n2 * 16 + (mi >> 1) * 8), kl);
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          const int n = 2 * n2 + y;
          const float d0 = btot[n * 8 + 2 * t], d1 = btot[n * 8 + 2 * t + 1];
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            S[m][n][0] *= d0;
            S[m][n][1] *= d1;
            S[m][n][2] *= d0;
            S[m][n][3] *= d1;
            la_mma(S[m][n], va[m], kh[2 * y], kh[2 * y + 1]);
            la_mma(S[m][n], va[m], kl[2 * y], kl[2 * y + 1]);
          }
        }
      }
    }
    __syncthreads();
  }
  float* dst = OUT ? st : cs;
  if ((!OUT || c == c_end - 1) && wlive) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int v = v0 + m * 16 + g + (e >> 1) * 8, k = n * 8 + 2 * t + (e & 1);
          if (v < a.dv && k < a.dk) dst[(long)k * a.dv + v] = S[m][n][e];
        }
  }
  if (!OUT && ch) a.total[((long)c * a.H + h) * a.dk + tid] = prod;
}

// dec[row][c] = sigmoid(W a + bias)^inv_tau. grid (channels / 128, rows / kDecayRows): thread = channel, the low-rank rows in shared
// memory, the channel's weights in registers (RK >= rank, a multiple of four) or, RK 0, in shared memory.
constexpr int kDecayRows = 32;
template <int RK, typename X>
__global__ void __launch_bounds__(128) linattn_decay_kernel(const X* __restrict__ a, long lda, const float* __restrict__ w, const float* __restrict__ bias,
                                                            float* __restrict__ dec, int rows, int C, int rank, float inv_tau) {
  extern __shared__ __align__(16) float ds[];             // [kDecayRows][RP], then (RK 0) [128][rank + 1]
  const int RP = RK ? RK : rank, c0 = blockIdx.x * 128, c = c0 + threadIdx.x, r0 = blockIdx.y * kDecayRows, n = min(kDecayRows, rows - r0);
  float* ws = ds + kDecayRows * RP;
  float wr[RK ? RK : 1];
  if (RK) {
#pragma unroll
    for (int r = 0; r < RK; ++r) wr[r] = r < rank && c < C ? w[(long)c * rank + r] : 0.f;
  } else {
    for (int i = threadIdx.x; i < 128 * rank; i += 128) ws[(i / rank) * (rank + 1) + i % rank] = c0 + i / rank < C ? w[(long)c0 * rank + i] : 0.f;
  }
  grid_dep_wait();
  grid_dep_launch();
  for (int i = threadIdx.x; i < n * RP; i += 128) {
    const int y = i / RP, r = i % RP;
    ds[i] = r < rank ? to_f(a[(long)(r0 + y) * lda + r]) : 0.f;
  }
  __syncthreads();
  if (c >= C) return;
  const float b = bias[c];
#pragma unroll 4
  for (int y = 0; y < n; ++y) {
    float z = b, z1 = 0.f, z2 = 0.f, z3 = 0.f;
    if (RK) {
#pragma unroll
      for (int r = 0; r < RK; r += 4) {
        const float4 v = *reinterpret_cast<const float4*>(ds + y * RK + r);
        z = fmaf(wr[RK ? r : 0], v.x, z);
        z1 = fmaf(wr[RK ? r + 1 : 0], v.y, z1);
        z2 = fmaf(wr[RK ? r + 2 : 0], v.z, z2);
        z3 = fmaf(wr[RK ? r + 3 : 0], v.w, z3);
      }
    } else {
      for (int r = 0; r < rank; ++r) z = fmaf(ws[threadIdx.x * (rank + 1) + r], ds[y * rank + r], z);
    }
    dec[(long)(r0 + y) * C + c] = root_decay((z + z1) + (z2 + z3), inv_tau);
  }
}

// Contributions -> start states, segment by segment (segments of one chunk have neither). grid (element blocks, H, segments).
__global__ void __launch_bounds__(256) linattn_scan_kernel(const LinChunkArgs a) {
  grid_dep_wait();
  grid_dep_launch();
  const int h = blockIdx.y, seg = blockIdx.z, c0 = a.seg_chunk0[seg], c1 = a.seg_chunk0[seg + 1];
  if (c1 - c0 < 2) return;
  const int first = a.chunk_first[c0], slot = a.slot[first], per = a.dk * a.dv, i = blockIdx.x * 256 + threadIdx.x;
  if (slot < 0 || i >= per) return;
  const int k = i / a.dv;
  float s = a.pos[first] != 0 ? a.state[((long)slot * a.H + h) * per + i] : 0.f;
  for (int c = c0; c < c1; ) {
    float u[8], d[8];
    const int n = min(8, c1 - c);
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (j < n && c + j < c1 - 1) {                      // the last chunk has no contribution
        u[j] = a.start[((long)(c + j) * a.H + h) * per + i];
        d[j] = a.total[((long)(c + j) * a.H + h) * a.dk + k];
      }
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (j < n) {
        a.start[((long)(c + j) * a.H + h) * per + i] = s;
        if (c + j < c1 - 1) s = fmaf(s, d[j], u[j]);
      }
    c += n;
  }
}

template <int DK, int DV, int MODE>
static int launch_chunks(const LinChunkArgs& a, int chunks, int segs, int longest, cudaStream_t st) {
  constexpr int base = (2 * 16 * ((MODE == 2 ? 3 : 2) * DK + DV) + (MODE == 2 ? 1 : 17) * DK) * 4 + 2 * 16 * (DK + 8) * 2 + 16 * (DV + 8) * 2;
  constexpr int full = base + 2 * 16 * (DK + 8) * 2 + 2 * 16 * 24 * 2 + 8 * 16 * 17 * 4 + (MODE == 2 ? 0 : 2 * 16 * DK * 4);
  static_assert(full <= 227 * 1024, "shared memory budget");
  static bool attr_set = false;
  if (!attr_set) {
    cudaError_t e = cudaFuncSetAttribute(linattn_chunk_kernel<DK, DV, MODE, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, full);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(linattn_chunk_kernel<DK, DV, MODE, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, full);
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  if (longest > 1) {
    launch_pdl(linattn_chunk_kernel<DK, DV, MODE, false>, dim3(chunks, a.H), dim3(128), base, st, a);
    launch_pdl(linattn_scan_kernel, dim3((a.dk * a.dv + 255) / 256, a.H, segs), dim3(256), 0, st, a);
  }
  launch_pdl(linattn_chunk_kernel<DK, DV, MODE, true>, dim3(chunks, a.H), dim3(128), full, st, a);
  return (int)cudaGetLastError();
}

}  // namespace ve

using namespace ve;

extern "C" {

// mode 0 / 1 / 2 as above (bias / lower, decay, or bias / w2 / rank / a_col / inv_tau / q_scale accordingly; plain: q_scale too). x32: the projection rows are fp32 (else bf16). nseg > 0: segment
// table; 0: segments from the slots of the rows (a few rows only: every CTA scans them).
int ve_linattn_step(const void* proj, long ld, int x32, const void* pos, const void* slot, const void* seg_first, const void* seg_count, int nseg,
                    void* state, const void* bias, const void* lower, const void* decay, void* o, long ldo, int rows, int H, int dk, int dv,
                    int mode, const void* w2, int rank, int a_col, float inv_tau, float q_scale, int plain, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (dk < 1 || dk > 256 || dv < 1 || H < 1 || (mode == 0 ? !decay : mode == 1 ? !bias || !lower : !bias || !w2 || rank < 1)) return cudaErrorInvalidValue;
  if (mode == 2 && rank % 4 == 0 && ((uintptr_t)w2 & 15)) return cudaErrorInvalidValue;
  LinArgs a{proj, ld, (const int*)pos, (const int*)slot, nseg > 0 ? (const int*)seg_first : nullptr, (const int*)seg_count, (float*)state,
            (const float*)bias, (const float*)lower, (const float*)decay, (float*)o, ldo, rows, H, dk, dv, (const float*)w2, rank, a_col, inv_tau, q_scale, plain};
  const dim3 grid(H, (dv + 31) / 32, nseg > 0 ? nseg : rows), block(32, 8);
#define VE_LS(NK, X, MODE) launch_pdl(linattn_step_kernel<NK, X, MODE>, grid, block, 0, st, a)
#define VE_LS_M(NK, X) do { if (mode == 0) VE_LS(NK, X, 0); else if (mode == 1) VE_LS(NK, X, 1); else VE_LS(NK, X, 2); } while (0)
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

// Decays of mode 2 for rows a [rows][rank] (pitch lda; fp32 when x32, else bf16), weights w [C][rank].
int ve_linattn_decay(const void* a, long lda, int x32, const void* w, const void* bias, void* dec, int rows, int C, int rank, float inv_tau, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (C < 1 || rank < 1 || rank > 320) return cudaErrorInvalidValue;         // (weights of 128 channels in shared memory above 32)
  const dim3 grid((C + 127) / 128, (rows + kDecayRows - 1) / kDecayRows);
  const int rk = rank <= 16 ? 16 : rank <= 32 ? 32 : 0;
  const size_t smem = (size_t)(kDecayRows * (rk ? rk : rank) + (rk ? 0 : 128 * (rank + 1))) * 4;
#define VE_LD(RK, X) do { \
    if (smem > 48 * 1024) { \
      const cudaError_t e = cudaFuncSetAttribute(linattn_decay_kernel<RK, X>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (e != cudaSuccess) return (int)e; \
    } \
    launch_pdl(linattn_decay_kernel<RK, X>, grid, dim3(128), smem, st, (const X*)a, lda, (const float*)w, (const float*)bias, (float*)dec, rows, C, rank, inv_tau); \
  } while (0)
#define VE_LD_R(X) do { if (rk == 16) VE_LD(16, X); else if (rk == 32) VE_LD(32, X); else VE_LD(0, X); } while (0)
  if (x32) VE_LD_R(float);
  else VE_LD_R(__nv_bfloat16);
#undef VE_LD_R
#undef VE_LD
  VE_CHECK_LAUNCH();
}

// The chunked form over a table of chunks (chunk_count <= 128 rows each; a segment's chunks follow each other, all but its last
// one a multiple of 16 rows): proj fp32, dk and dv <= 128. start / total: scratch (see LinChunkArgs); longest: most chunks of
// any segment.
int ve_linattn_chunk(const void* proj, long ld, const void* pos, const void* slot, const void* chunk_seg, const void* chunk_first, const void* chunk_count,
                     const void* seg_chunk0, int chunks, int segs, int longest, void* state, void* start, void* total, const void* bias, const void* lower,
                     const void* decay, void* o, long ldo, int H, int dk, int dv, int mode, const void* dec, float q_scale, int plain, cudaStream_t st) {
  if (chunks <= 0) return 0;
  if (mode == 2 && !dec) return cudaErrorInvalidValue;
  if (dk < 1 || dk > 128 || dv < 1 || dv > 128 || H < 1 || segs < 1 || (mode == 0 ? !decay : mode == 1 && (!bias || !lower))) return cudaErrorInvalidValue;
  const int vec = !((uintptr_t)proj & 15) && ld % 4 == 0 && dk % 4 == 0 && dv % 4 == 0 && !((uintptr_t)dec & 15);
  LinChunkArgs a{(const float*)proj, ld, (const int*)pos, (const int*)slot, (const int*)chunk_seg, (const int*)chunk_first, (const int*)chunk_count,
                 (const int*)seg_chunk0, (float*)state, (float*)start, (float*)total, (const float*)bias, (const float*)lower, (const float*)decay,
                 (float*)o, ldo, H, dk, dv, vec, (const float*)dec, q_scale, plain};
#define VE_LC(DK, DV) return mode == 0 ? launch_chunks<DK, DV, 0>(a, chunks, segs, longest, st) : mode == 1 ? launch_chunks<DK, DV, 1>(a, chunks, segs, longest, st) \
    : launch_chunks<DK, DV, 2>(a, chunks, segs, longest, st)
#define VE_LC_V(DK) do { if (dv <= 32) VE_LC(DK, 32); if (dv <= 64) VE_LC(DK, 64); VE_LC(DK, 128); } while (0)
  if (dk <= 32) VE_LC_V(32);
  if (dk <= 64) VE_LC_V(64);
  VE_LC_V(128);
#undef VE_LC_V
#undef VE_LC
}

}  // extern "C"
