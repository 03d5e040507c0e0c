// bf16 linears on a few rows (decode / verify steps), with the step in front in the prologue and the step behind in the
// epilogue, for decoders with an fp32 residual stream:
//   y[m][n] = sum_k W[n][k] x[m][k],   m < 16
//   prologue   0  x given in bf16
//              1  x = tanh(alpha h) w + b of the fp32 residual h
//              2  x = RMS norm over groups of columns of an fp32 row [* sigmoid(gate) or silu(gate)], behind columns taken as they are
//              3  x = PolyNorm of an fp32 row
//              4  x = layer norm (no shift) of the weighted sum of the fp32 residual streams
//              5  x = clamped gated unit of an fp32 [gate | up] row
//              6  x = h + RMS norm of a sublayer's result (fp32, optional), as it is or RMS normed; the sum is also stored
//              (the row that enters the product can be stored too, in bf16)
//   epilogue   add a bias (optional), then store fp32 (with a soft cap or without) or bf16, or h += scale * y on the fp32 residual, or the residual streams rewritten (streams_write), or, for
//              weight rows in blocks of [4 gate | 4 up], the clamped gated unit of the pairs in bf16 (half as many columns)
// The rows are the M side (16) of mma.sync.m16n8k16 and eight weight rows the N side. The order of k inside a product does
// not matter, so a lane takes eight consecutive k of one weight row as 16 bytes and uses them as the B operands of two MMAs, the
// matching activations as the A operands. Weights are read once; the first of them are requested before the programmatic
// dependency wait, so they arrive while the kernel in front finishes.
// gemm_f32 is the plain fp32 product of the all-32-bit form.
#include "rowmath.cuh"

namespace ve {

struct RowsArgs {
  const __nv_bfloat16* W; long ldw;
  int N, K, M;                      // K: columns of W (a multiple of 8)
  int pro, kx;                      // kx <= K: columns of x (the rest read as zero)
  const void* x; long ldx;
  const float* w; const float* b; float alpha;
  int G, wlen;
  const float* gate; long ldg;
  const float* coef; float eps;
  float* out_f32; __nv_bfloat16* out; long ldo;
  float* h; long ldh; const float* scale;
  const float* head; long ldhead; int k0;     // prologue 2: the first k0 columns of x, as they are
  int silu;                         // prologue 2: activation of the gate
  int glu; Glu unit;                // epilogue (and prologue 5)
  float cap;                        // > 0: soft cap of the fp32 output
  const float* part; long ldpart; float* h_out;          // prologue 6: w normalises part, b the sum (null: none); h_out [M][kx]
  __nv_bfloat16* x_out;             // prologue 6: the rows that enter the product, [M][kx] (null: not stored)
  const float* bias;                // [N] (null: none)
  int v4;                           // prologue 6: four columns at a time
  int streams; const float* hmix;   // streams > 0: h [M][streams][N], scale [streams]
  int pitch;                        // bytes per activation row in shared memory (prologue forms)
};

VE_DEVINL void rows_mma(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

VE_DEVINL void rows_out(const RowsArgs& a, int m, int n, float v) {
  if (a.streams) {
    float* hp = a.h + m * a.ldh + n;
    float x[kMaxStreams];
#pragma unroll
    for (int s = 0; s < kMaxStreams; ++s) x[s] = s < a.streams ? hp[(long)s * a.N] : 0.f;
    streams_write(x, a.streams, a.hmix, a.scale, v);
#pragma unroll
    for (int s = 0; s < kMaxStreams; ++s)
      if (s < a.streams) hp[(long)s * a.N] = x[s];
  } else if (a.h) a.h[m * a.ldh + n] = fmaf(v, a.scale ? a.scale[n] : 1.f, a.h[m * a.ldh + n]);
  else if (a.out_f32) a.out_f32[m * a.ldo + n] = a.cap > 0.f ? soft_cap_of(v, a.cap) : v;
  else a.out[m * a.ldo + n] = f2bf(v);
}

template <int V> struct Cols;
template <> struct Cols<1> {
  float v[1];
  VE_DEVINL void load(const float* p) { v[0] = *p; }
  VE_DEVINL void store(float* p) const { *p = v[0]; }
  VE_DEVINL void store(__nv_bfloat16* p) const { *p = f2bf(v[0]); }
};
template <> struct Cols<4> {
  float v[4];
  VE_DEVINL void load(const float* p) {
    const float4 t = load4(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  }
  VE_DEVINL void store(float* p) const { store4(p, make_float4(v[0], v[1], v[2], v[3])); }
  VE_DEVINL void store(__nv_bfloat16* p) const { store4(p, make_float4(v[0], v[1], v[2], v[3])); }
};

// Prologue 6: one exchange between the warps for all rows and norm. The first CTA stores the sum.
template <int V>
VE_DEVINL void residual_prologue(const RowsArgs& a, uint8_t* xs, float* red) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const float* h = reinterpret_cast<const float*>(a.x);
  auto gather = [&](float s, int m, float* r) {
    s = warp_sum(s);
    if (lane == 0) r[m * 8 + warp] = s;
  };
  auto over = [&](int m, const float* r) {
    float s = 0.f;
#pragma unroll
    for (int y = 0; y < 8; ++y) s += r[m * 8 + y];
    return 1.f / sqrtf(s / (float)a.kx + a.eps);
  };
  auto sum = [&](int m, int i, float inv, Cols<V>& x) {
    x.load(h + m * a.ldx + i);
    if (!a.part) return;
    Cols<V> y, w;
    y.load(a.part + m * a.ldpart + i);
    w.load(a.w + i);
#pragma unroll
    for (int e = 0; e < V; ++e) x.v[e] = fmaf(y.v[e] * inv, w.v[e], x.v[e]);
  };
  if (a.part) {
    for (int m = 0; m < a.M; ++m) {
      float s = 0.f;
#pragma unroll 4
      for (int i = tid * V; i < a.kx; i += 256 * V) {
        Cols<V> y;
        y.load(a.part + m * a.ldpart + i);
#pragma unroll
        for (int e = 0; e < V; ++e) s = fmaf(y.v[e], y.v[e], s);
      }
      gather(s, m, red);
    }
    __syncthreads();
  }
  if (a.b) {
    for (int m = 0; m < a.M; ++m) {
      const float inv = a.part ? over(m, red) : 0.f;
      float s = 0.f;
#pragma unroll 4
      for (int i = tid * V; i < a.kx; i += 256 * V) {
        Cols<V> x;
        sum(m, i, inv, x);
#pragma unroll
        for (int e = 0; e < V; ++e) s = fmaf(x.v[e], x.v[e], s);
      }
      gather(s, m, red + 64);
    }
    __syncthreads();
  }
  for (int m = 0; m < a.M; ++m) {
    const float inv = a.part ? over(m, red) : 0.f, inv2 = a.b ? over(m, red + 64) : 1.f;
    __nv_bfloat16* xr = reinterpret_cast<__nv_bfloat16*>(xs + m * a.pitch);
#pragma unroll 4
    for (int i = tid * V; i < a.kx; i += 256 * V) {
      Cols<V> x;
      sum(m, i, inv, x);
      if (a.h_out && blockIdx.x == 0) x.store(a.h_out + (long)m * a.kx + i);
      if (a.b) {
        Cols<V> w;
        w.load(a.b + i);
#pragma unroll
        for (int e = 0; e < V; ++e) x.v[e] *= inv2 * w.v[e];
      }
      x.store(xr + i);
      if (a.x_out && blockIdx.x == 0) x.store(a.x_out + (long)m * a.kx + i);
    }
  }
}

// Activations of the prologue forms -> bf16 rows in shared memory.
VE_DEVINL void rows_prologue(const RowsArgs& a, uint8_t* xs, float* red) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, K32 = (a.K + 31) / 32 * 32;
  const float* src = reinterpret_cast<const float*>(a.x);
  auto put = [&](int m, int k, float v) { reinterpret_cast<__nv_bfloat16*>(xs + m * a.pitch)[k] = f2bf(v); };
  for (int i = a.kx + tid; i < K32; i += 256)
    for (int m = 0; m < a.M; ++m) put(m, i, 0.f);
  if (a.pro == 1) {
    for (int k = tid; k < a.kx; k += 256) {
      const float wk = a.w[k], bk = a.b[k];
      for (int m = 0; m < a.M; ++m) put(m, k, dyt_of(src[m * a.ldx + k], a.alpha, wk, bk));
    }
  } else if (a.pro == 2) {
    const int groups = (a.kx - a.k0) / a.G;
    for (int i = tid; i < a.k0; i += 256)
      for (int m = 0; m < a.M; ++m) put(m, i, a.head[m * a.ldhead + i]);
    if (groups * a.M >= 8) {
      for (int p = warp; p < groups * a.M; p += 8) {
        const int m = p / groups, c0 = (p % groups) * a.G;
        float ss = 0.f;
        for (int i = lane; i < a.G; i += 32) {
          const float v = src[m * a.ldx + c0 + i];
          ss = fmaf(v, v, ss);
        }
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)a.G + a.eps);
        for (int i = lane; i < a.G; i += 32) {
          const int c = c0 + i;
          float v = src[m * a.ldx + c] * inv * a.w[c % a.wlen];
          if (a.gate) v *= a.silu ? silu_of(a.gate[m * a.ldg + c]) : sigmoid_of(a.gate[m * a.ldg + c]);
          put(m, a.k0 + c, v);
        }
      }
    } else {
      for (int p = 0; p < groups * a.M; ++p) {
        const int m = p / groups, c0 = (p % groups) * a.G;
        float ss = 0.f;
        for (int i = tid; i < a.G; i += 256) {
          const float v = src[m * a.ldx + c0 + i];
          ss = fmaf(v, v, ss);
        }
        const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)a.G + a.eps);
        for (int i = tid; i < a.G; i += 256) {
          const int c = c0 + i;
          float v = src[m * a.ldx + c] * inv * a.w[c % a.wlen];
          if (a.gate) v *= a.silu ? silu_of(a.gate[m * a.ldg + c]) : sigmoid_of(a.gate[m * a.ldg + c]);
          put(m, a.k0 + c, v);
        }
      }
    }
  } else if (a.pro == 4) {
    // sums of every row around its first column (so that a common offset does not cancel digits), one exchange for all rows
    const int S = a.G;
    float win[kMaxStreams];
#pragma unroll
    for (int s = 0; s < kMaxStreams; ++s) win[s] = s < S ? a.coef[s] : 0.f;
    auto read = [&](int m, int k) {
      float u = 0.f;
#pragma unroll
      for (int s = 0; s < kMaxStreams; ++s)
        if (s < S) u = fmaf(win[s], src[m * a.ldx + (long)s * a.kx + k], u);
      return u;
    };
    for (int m = 0; m < a.M; ++m) {
      const float c = read(m, 0);
      float s1 = 0.f, s2 = 0.f;
      for (int i = tid; i < a.kx; i += 256) {
        const float d = read(m, i) - c;
        s1 += d;
        s2 = fmaf(d, d, s2);
      }
      s1 = warp_sum(s1);
      s2 = warp_sum(s2);
      if (lane == 0) {
        red[(m * 8 + warp) * 2] = s1;
        red[(m * 8 + warp) * 2 + 1] = s2;
      }
    }
    __syncthreads();
    for (int m = 0; m < a.M; ++m) {
      const float c = read(m, 0), n = 1.f / (float)a.kx;
      float s1 = 0.f, s2 = 0.f;
#pragma unroll
      for (int y = 0; y < 8; ++y) {
        s1 += red[(m * 8 + y) * 2];
        s2 += red[(m * 8 + y) * 2 + 1];
      }
      const float d = s1 * n, inv = 1.f / sqrtf(fmaxf(fmaf(-d, d, s2 * n), 0.f) + a.eps);
      for (int i = tid; i < a.kx; i += 256) put(m, i, (read(m, i) - c - d) * inv * a.w[i]);
    }
  } else if (a.pro == 5) {
    for (int m = 0; m < a.M; ++m)
      for (int i = tid; i < a.kx; i += 256) put(m, i, clamped_glu_of(src[m * a.ldx + i], src[m * a.ldx + a.kx + i], a.unit));
  } else if (a.pro == 6) {
    if (a.v4) residual_prologue<4>(a, xs, red);
    else residual_prologue<1>(a, xs, red);
  } else {
    for (int m = 0; m < a.M; ++m) {
      float s1 = 0.f, s2 = 0.f, s3 = 0.f;
      for (int i = tid; i < a.kx; i += 256) poly_sums(src[m * a.ldx + i], s1, s2, s3);
      s1 = warp_sum(s1);
      s2 = warp_sum(s2);
      s3 = warp_sum(s3);
      __syncthreads();                                     // (readers of the row in front)
      if (lane == 0) {
        red[warp] = s1;
        red[33 + warp] = s2;
        red[66 + warp] = s3;
      }
      __syncthreads();
      s1 = s2 = s3 = 0.f;
#pragma unroll
      for (int y = 0; y < 8; ++y) {
        s1 += red[y];
        s2 += red[33 + y];
        s3 += red[66 + y];
      }
      const PolyScale ps = poly_scale(s1, s2, s3, a.kx, a.eps, a.coef);
      for (int i = tid; i < a.kx; i += 256) put(m, i, poly_of(src[m * a.ldx + i], ps));
    }
  }
  __syncthreads();
}

// All activations in shared memory (made by the prologue, or copied). Resident CTAs (two per SM) walk tiles of eight weight rows; the
// eight warps of a CTA share the k of a tile in units of 32 k. Every lane copies the 16-byte pieces it will use itself into a ring of its
// own in shared memory (cp.async, groups of four units, DEPTH groups), so no barrier stands between the copies and their use and
// nothing waits in order for younger loads. The first groups are requested before the dependency wait. HI: more than eight rows.
template <int DEPTH, bool HI>
__global__ void __launch_bounds__(256, 2) gemv_ring_kernel(const RowsArgs a) {
  constexpr int U = 4, GROUP = 8 * U * 512;               // bytes of one group of all warps
  extern __shared__ __align__(16) uint8_t xs[];           // [M][pitch] activations, then [DEPTH][8 warps][U][32 lanes][16 B]
  __shared__ float part[8][8][HI ? 16 : 8][8], red[4][33];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  uint8_t* ring = xs + a.M * a.pitch + (warp * U * 32 + lane) * 16;
  const uint32_t ring_s = smem_u32(ring);
  const int tiles = (a.N + 7) / 8, units = (a.K + 31) / 32, per_tile = (units + 8 * U - 1) / (8 * U);      // groups per tile
  const int mine = (tiles - (int)blockIdx.x + (int)gridDim.x - 1) / (int)gridDim.x, total = mine * per_tile;
  // unit of the group's j-th place: neighbours are halves of one 128-byte line of a weight row
  auto unit_of = [&](int gi, int j) { return ((gi * (U / 2) + (j >> 1)) * 8 + warp) * 2 + (j & 1); };
  int i_tile = blockIdx.x, i_g = 0, i_stage = 0, i_left = total;      // what is requested next
  auto issue = [&]() {
    if (i_left > 0) {
      const __nv_bfloat16* wr = a.W + (long)min(i_tile * 8 + g, a.N - 1) * a.ldw + t * 8;
#pragma unroll
      for (int j = 0; j < U; ++j) {
        const int u = unit_of(i_g, j);
        const bool in = u * 32 + t * 8 < a.K;
        const int n = in ? 16 : 0;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(ring_s + i_stage * GROUP + j * 512), "l"(in ? wr + u * 32 : a.W), "r"(n) : "memory");
      }
      --i_left;
      if (++i_g == per_tile) {
        i_g = 0;
        i_tile += gridDim.x;
      }
      if (++i_stage == DEPTH) i_stage = 0;
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int d = 0; d < DEPTH - 1; ++d) issue();
  grid_dep_wait();
  grid_dep_launch();
  if (a.pro) {
    rows_prologue(a, xs, &red[0][0]);
  } else {
    const __nv_bfloat16* xg = reinterpret_cast<const __nv_bfloat16*>(a.x);
    const int K32 = units * 32;
    for (int i = tid; i < a.M * (K32 / 8); i += 256) {
      const int m = i / (K32 / 8), k = (i % (K32 / 8)) * 8;
      *reinterpret_cast<uint4*>(xs + m * a.pitch + k * 2) = k < a.K ? *reinterpret_cast<const uint4*>(xg + m * a.ldx + k) : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();
  }
  float c[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) c[i][0] = c[i][1] = c[i][2] = c[i][3] = 0.f;
  const bool lo_in = g < a.M, hi_in = HI && g + 8 < a.M;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  const uint8_t* xlo = xs + g * a.pitch + t * 16;
  int stage = 0, gi = 0, done = 0;                        // done: tiles finished
  for (int it = 0; it < total; ++it) {
    issue();                                              // into the stage the group in front was read from
    asm volatile("cp.async.wait_group %0;" ::"n"(DEPTH - 1) : "memory");
    uint4 w[U], lo[U], hi[U];
#pragma unroll
    for (int j = 0; j < U; ++j) {
      const int u = unit_of(gi, j);
      w[j] = *reinterpret_cast<const uint4*>(ring + stage * GROUP + j * 512);
      lo[j] = lo_in && u < units ? *reinterpret_cast<const uint4*>(xlo + u * 64) : zero;
      hi[j] = hi_in && u < units ? *reinterpret_cast<const uint4*>(xlo + 8 * a.pitch + u * 64) : zero;
    }
#pragma unroll
    for (int j = 0; j < U; ++j) {
      rows_mma(c[j & 1], lo[j].x, hi[j].x, lo[j].y, hi[j].y, w[j].x, w[j].y);
      rows_mma(c[2 + (j & 1)], lo[j].z, hi[j].z, lo[j].w, hi[j].w, w[j].z, w[j].w);
    }
    if (++stage == DEPTH) stage = 0;
    if (++gi < per_tile) continue;
    gi = 0;
    // The warps' sums of this tile go to one of eight buffers; the warps take turns adding them up while the others go on. A
    // buffer comes round after eight tiles, and every warp has waited for all others once in between.
    const int buf = done & 7, bar = 1 + buf;
    float* pt = &part[buf][warp][0][0];
    pt[g * 8 + 2 * t] = (c[0][0] + c[1][0]) + (c[2][0] + c[3][0]);
    pt[g * 8 + 2 * t + 1] = (c[0][1] + c[1][1]) + (c[2][1] + c[3][1]);
    if (HI) {
      pt[(g + 8) * 8 + 2 * t] = (c[0][2] + c[1][2]) + (c[2][2] + c[3][2]);
      pt[(g + 8) * 8 + 2 * t + 1] = (c[0][3] + c[1][3]) + (c[2][3] + c[3][3]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) c[i][0] = c[i][1] = c[i][2] = c[i][3] = 0.f;
    if (buf != warp) {
      asm volatile("bar.arrive %0, 256;" ::"r"(bar) : "memory");
    } else {
      asm volatile("bar.sync %0, 256;" ::"r"(bar) : "memory");
      const int n0 = (blockIdx.x + done * gridDim.x) * 8;
      for (int i0 = 0; i0 < a.M * 8; i0 += 32) {
        const int i = i0 + lane;
        const bool in = i < a.M * 8 && n0 + (i & 7) < a.N;
        float v = 0.f;
        if (in)
#pragma unroll
          for (int y = 0; y < 8; ++y) v += (&part[buf][y][0][0])[i];
        if (in && a.bias) v += a.bias[n0 + (i & 7)];
        if (a.glu) {                                      // lanes e and e + 4 of a row hold a pair
          const float u = __shfl_down_sync(0xffffffffu, v, 4);
          if (in && (i & 7) < 4) a.out[(i >> 3) * a.ldo + n0 / 2 + (i & 3)] = f2bf(clamped_glu_of(v, u, a.unit));
        } else if (in) {
          rows_out(a, i >> 3, n0 + (i & 7), v);
        }
      }
    }
    ++done;
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
}

// Rows whose activations do not fit: they pass through shared memory in slabs of eight units per slice of k. 8 warps: R tiles of 8
// weight rows x KS slices of k, weights from global memory to registers (a ring of eight 16-byte loads per lane).
template <int KS, bool HI>
__global__ void __launch_bounds__(256, 3) gemv_slab_kernel(const RowsArgs a) {
  constexpr int R = 8 / KS, PF = 8, SLAB = KS * PF * 32, SP = SLAB * 2 + 64;
  extern __shared__ __align__(16) uint8_t xs[];
  __shared__ float part[2][8][HI ? 16 : 8][8];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int ks = warp % KS, rt = warp / KS;
  const int units = (a.K + 31) / 32, batches = ((units + KS - 1) / KS + PF - 1) / PF;
  const int groups = ((a.N + 7) / 8 + R - 1) / R;
  auto row_of = [&](int grp) { return a.W + (long)min((grp * R + rt) * 8 + g, a.N - 1) * a.ldw + t * 8; };
  auto load_w = [&](const __nv_bfloat16* wr, int u, bool in) -> uint4 {
    if (in && u * 32 + t * 8 < a.K) return __ldcs(reinterpret_cast<const uint4*>(wr + u * 32));
    return make_uint4(0, 0, 0, 0);
  };
  int grp = blockIdx.x;
  uint4 buf[PF];
  {
    const __nv_bfloat16* wr = row_of(grp);
#pragma unroll
    for (int j = 0; j < PF; ++j) buf[j] = load_w(wr, ks + j * KS, true);
  }
  grid_dep_wait();
  grid_dep_launch();
  const __nv_bfloat16* xg = reinterpret_cast<const __nv_bfloat16*>(a.x);
  auto slab = [&](int b, int stage) {                     // activations of batch b -> xs[stage]
    constexpr int C8 = SLAB / 8;
    for (int i = tid; i < (HI ? 16 : 8) * C8; i += 256) {
      const int m = i / C8, k = b * SLAB + (i % C8) * 8;
      const bool in = m < a.M && k < a.K;
      const int n = in ? 16 : 0;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(xs + (stage * (HI ? 16 : 8) + m) * SP + (i % C8) * 16)),
                   "l"(xg + (in ? m * a.ldx + k : 0)), "r"(n) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  slab(0, 0);
  int pb = 0, stage = 0;
  for (; grp < groups; grp += gridDim.x) {
    float c[4] = {0.f, 0.f, 0.f, 0.f};
    for (int b = 0; b < batches; ++b) {
      const bool last = b + 1 == batches;
      const int ngrp = last ? grp + gridDim.x : grp, nu = last ? ks : ks + (b + 1) * PF * KS;
      const __nv_bfloat16* wr = row_of(ngrp);
      if (!last || ngrp < groups) {
        slab(last ? 0 : b + 1, stage ^ 1);
        asm volatile("cp.async.wait_group 1;" ::: "memory");
      } else {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
      }
      __syncthreads();
#pragma unroll
      for (int j = 0; j < PF; ++j) {
        const uint4 w = buf[j];
        buf[j] = load_w(wr, nu + j * KS, ngrp < groups);
        const int u = ks + (b * PF + j) * KS;
        if (u < units) {
          uint4 lo = make_uint4(0, 0, 0, 0), hi = make_uint4(0, 0, 0, 0);
          const uint8_t* p = xs + (stage * (HI ? 16 : 8) + g) * SP + (j * KS + ks) * 64 + t * 16;
          lo = *reinterpret_cast<const uint4*>(p);
          if (HI) hi = *reinterpret_cast<const uint4*>(p + 8 * SP);
          rows_mma(c, lo.x, hi.x, lo.y, hi.y, w.x, w.y);
          rows_mma(c, lo.z, hi.z, lo.w, hi.w, w.z, w.w);
        }
      }
      stage ^= 1;
      __syncthreads();                                    // the slab behind may be overwritten now
    }
    part[pb][warp][g][2 * t] = c[0];
    part[pb][warp][g][2 * t + 1] = c[1];
    if (HI) {
      part[pb][warp][(HI ? 8 : 0) + g][2 * t] = c[2];
      part[pb][warp][(HI ? 8 : 0) + g][2 * t + 1] = c[3];
    }
    __syncthreads();
    for (int i = tid; i < a.M * R * 8; i += 256) {
      const int m = i / (R * 8), q = i % (R * 8), r = q / 8, e = q % 8, n = (grp * R + r) * 8 + e;
      if (n >= a.N) continue;
      float v = 0.f;
#pragma unroll
      for (int s = 0; s < KS; ++s) v += part[pb][r * KS + s][m][e];
      if (a.bias) v += a.bias[n];
      rows_out(a, m, n, v);
    }
    pb ^= 1;                                              // (the other buffer's readers are done: they passed the barrier above)
  }
}

// out[t][n] = sum_k W[n][k] x[t][k] (+ bias[n]), fp32 throughout. 64 x 64 tiles, 16 k per step, 4 x 4 outputs per thread.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ W, long ldw, const float* __restrict__ x, long ldx, float* __restrict__ out,
                                                       long ldo, int T, int N, int K, const float* __restrict__ bias) {
  __shared__ float sw[16][65], sx[16][65];
  const int tid = threadIdx.x, n0 = blockIdx.x * 64, t0 = blockIdx.y * 64, tn = (tid & 15) * 4, tt = (tid >> 4) * 4;
  grid_dep_wait();
  grid_dep_launch();
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int i = tid; i < 64 * 16; i += 256) {
      const int r = i >> 4, k = i & 15;
      sw[k][r] = (n0 + r < N && k0 + k < K) ? W[(long)(n0 + r) * ldw + k0 + k] : 0.f;
      sx[k][r] = (t0 + r < T && k0 + k < K) ? x[(long)(t0 + r) * ldx + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(sx[k][tt + i], sw[k][tn + j], acc[i][j]);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (t0 + tt + i < T && n0 + tn + j < N) out[(long)(t0 + tt + i) * ldo + n0 + tn + j] = bias ? acc[i][j] + bias[n0 + tn + j] : acc[i][j];
}

template <typename F>
static int allow_smem(F kernel, int smem, int& have) {
  if (smem <= have) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e == cudaSuccess) have = smem;
  return (int)e;
}

template <int DEPTH, bool HI>
static int launch_ring_d(const RowsArgs& a, cudaStream_t st) {
  const int smem = a.M * a.pitch + DEPTH * 16 * 1024, tiles = (a.N + 7) / 8;
  static int have = 0;
  const int rc = allow_smem(gemv_ring_kernel<DEPTH, HI>, smem, have);
  if (rc) return rc;
  const int ctas = !HI && (smem + 18 * 1024) * 2 <= 227 * 1024 ? 296 : 148;
  launch_pdl(gemv_ring_kernel<DEPTH, HI>, dim3(tiles < ctas ? tiles : ctas), dim3(256), smem, st, a);
  return (int)cudaGetLastError();
}
template <bool HI>
static int launch_ring(const RowsArgs& a, cudaStream_t st) {
  const int room = (95 * 1024 - a.M * a.pitch) / (16 * 1024);           // groups that fit in half of the SM's shared memory
  if (room >= 5) return launch_ring_d<5, HI>(a, st);
  if (room == 4) return launch_ring_d<4, HI>(a, st);
  return launch_ring_d<3, HI>(a, st);
}

template <int KS, bool HI>
static int launch_slab(const RowsArgs& a, cudaStream_t st) {
  constexpr int smem = 2 * (HI ? 16 : 8) * (KS * 8 * 32 * 2 + 64);
  static int have = 0;
  const int rc = allow_smem(gemv_slab_kernel<KS, HI>, smem, have);
  if (rc) return rc;
  const int groups = ((a.N + 7) / 8 + 8 / KS - 1) / (8 / KS);
  const int per = (smem + (HI ? 9 : 5) * 1024) * 3 <= 222 * 1024 ? 3 : (smem + (HI ? 9 : 5) * 1024) * 2 <= 222 * 1024 ? 2 : 1;
  launch_pdl(gemv_slab_kernel<KS, HI>, dim3(groups < 148 * per ? groups : 148 * per), dim3(256), smem, st, a);
  return (int)cudaGetLastError();
}

}  // namespace ve

using namespace ve;

extern "C" {

// pro 0: x bf16 [M, K], M <= 16. pro 1..6: x fp32, M <= 8 and the activation rows (kx columns) fit in shared memory (else refused).
// pro 2 with k0 > 0: columns [0, k0) from head, the norm's columns behind them. pro 4: G streams of kx columns weighted by coef.
// pro 5: 2 kx columns, glu_alpha, glu_limit and glu_shift. pro 6: part fp32 (null: none) normed with w, the sum with b (null: not), stored to
// h_out [M][kx] (null: not), what enters the product to x_out [M][kx] (null: not). bias fp32 [N] (null: none). cap > 0: soft cap of out_f32. glu: out bf16 [M][N / 2] (N a multiple of 8). Exactly one of h, out_f32 and out is written; streams > 0: h [M][streams][N]
// with hmix [streams][streams] and scale [streams].
int ve_gemv_rows(const void* W, long ldw, int N, int K, int M, int pro, int kx, const void* x, long ldx, const void* w, const void* b, float alpha, int G,
                 int wlen, const void* gate, long ldg, const void* coef, float eps, void* out_f32, void* out, long ldo, void* h, long ldh, const void* scale,
                 const void* head, long ldhead, int k0, int silu, int glu, float glu_alpha, float glu_limit, float glu_shift, int streams, const void* hmix,
                 float cap, const void* part, long ldpart, void* h_out, void* x_out, const void* bias, cudaStream_t st) {
  if (M <= 0 || N <= 0) return 0;
  if (K % 8 || ldw % 8 || ((uintptr_t)W & 15) || M > 16 || kx > K || kx < 1 || pro < 0 || pro > 6) return cudaErrorInvalidValue;
  RowsArgs a{(const __nv_bfloat16*)W, ldw, N, K, M, pro, kx, x, ldx, (const float*)w, (const float*)b, alpha, G, wlen, (const float*)gate, ldg,
             (const float*)coef, eps, (float*)out_f32, (__nv_bfloat16*)out, ldo, (float*)h, ldh, (const float*)scale,
             (const float*)head, ldhead, k0, silu, glu, Glu{glu_alpha, glu_limit, glu_shift}, cap, (const float*)part, ldpart, (float*)h_out, (__nv_bfloat16*)x_out, (const float*)bias,
             kx % 4 == 0 && ldx % 4 == 0 && ldpart % 4 == 0 && !(((uintptr_t)x | (uintptr_t)part | (uintptr_t)w | (uintptr_t)b | (uintptr_t)h_out | (uintptr_t)x_out) & 15),
             streams, (const float*)hmix, 0};
  if (glu && (!out || N % 8 || (long)M * ((K + 31) / 32 * 64 + 64) > 100 * 1024)) return cudaErrorInvalidValue;
  if (streams < 0 || streams > kMaxStreams || (streams && (!h || !hmix || !scale))) return cudaErrorInvalidValue;
  const int K32 = (K + 31) / 32 * 32;
  a.pitch = K32 * 2 + ((K32 * 2) % 128 == 0 ? 64 : 0);            // rows of a quad pair land in different halves of the banks
  if (pro) {
    if (M > 8 || (long)M * a.pitch > 100 * 1024) return cudaErrorInvalidValue;
    if ((pro == 1 && (!w || !b || h)) || (pro == 2 && (!w || G < 1 || k0 < 0 || k0 > kx || (kx - k0) % G || wlen < 1 || (k0 && !head))) ||
        (pro == 3 && !coef) || (pro == 6 && part && !w) || (pro == 4 && (!w || !coef || G < 1 || G > kMaxStreams || h))) return cudaErrorInvalidValue;
  } else if (kx != K || ldx % 8 || ((uintptr_t)x & 15)) {
    return cudaErrorInvalidValue;
  }
  if ((long)M * a.pitch <= 100 * 1024) return M <= 8 ? launch_ring<false>(a, st) : launch_ring<true>(a, st);
  const int tiles = (N + 7) / 8;
#define VE_GR(KS) (M <= 8 ? launch_slab<KS, false>(a, st) : launch_slab<KS, true>(a, st))
  if (tiles >= 4 * 120) return VE_GR(2);
  if (tiles >= 2 * 120) return VE_GR(4);
  return VE_GR(8);
#undef VE_GR
}

int ve_gemm_f32(const void* W, long ldw, const void* x, long ldx, void* out, long ldo, int T, int N, int K, const void* bias, cudaStream_t st) {
  if (T <= 0 || N <= 0) return 0;
  launch_pdl(gemm_f32_kernel, dim3((N + 63) / 64, (T + 63) / 64), dim3(256), 0, st, (const float*)W, ldw, (const float*)x, ldx, (float*)out, ldo, T, N, K, (const float*)bias);
  VE_CHECK_LAUNCH();
}

}  // extern "C"
