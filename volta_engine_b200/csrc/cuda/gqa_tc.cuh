// Grouped-query attention of prompt rows on the fifth-generation tensor cores (tcgen05, accumulators in TMEM). Included by gqa.cu.
//
// One CTA = up to 128 packed rows ((token, head-in-group) pairs of one kv head) of one sequence against the pages of its cache. The
// structure is that of attention_tc.cuh (two streams of alternating pages, each with its own S buffers, softmax warps, running
// reference and O accumulator; lazy moves of the reference; merge in the epilogue) with these differences:
//   * query / key are DQC chunks of 64 columns, values DVC chunks (columns behind the real width are zero: the query's by the loader,
//     the pages' by the tensor map); keys and values have rings of their own (a key page is free as soon as its scores are done);
//   * a bias by distance is added to the scaled scores: one value per row for pages far enough back, a table look-up otherwise;
//   * the softmax weights enter the second product as two bf16 terms (value and remainder), so they keep 32-bit quality;
//   * with a sliding window the pages between the first tokens that stay in sight and the first token's window are not visited;
//   * a soft cap bends the scores in front of the bias (an exponential each and a quarter of a reciprocal: cap2_of4);
//   * the sink joins the sums in the epilogue, the result is turned back and gated there.
// Every wait is bounded; on expiry the CTA records a status code, skips its stores and frees its TMEM.
#pragma once

namespace ve {

struct GqaTc {
  GqaDims n;
  GqaRows rw;
  GqaScore sc;
  const __nv_bfloat16* q;                  // [rows][H][kw]
  const int* tile_first; const int* tile_count;
  __nv_bfloat16* out; long ldo;
  int vec;                                 // 16-byte stores are aligned
  int* status;
};

constexpr int kGtRows = 128, kGtThreads = 320;
constexpr float kGtLazyLog2 = 8.f;

// Page stages: a page's keys and values are requested in turn, and the values wait for the weights of their page; with four stages
// the requests run far enough ahead that no product waits for memory.
template <int DQC, int DVC> struct GtStages {
  static constexpr int K = DQC > 3 ? 2 : 4, V = DQC > 3 && DVC > 1 ? 2 : 4;
};

// Gates of eight columns from c on, of which `live` exist.
VE_DEVINL void gate8(const GqaScore& sc, long row, int c, int live, float* g) {
  if (!sc.gate) {
#pragma unroll
    for (int e = 0; e < 8; ++e) g[e] = 1.f;
  } else if (sc.gatev) {
    const long at = row * sc.ldg + c;
    float4 x, y;
    if (sc.gate32) {
      x = load4(reinterpret_cast<const float*>(sc.gate) + at);
      y = load4(reinterpret_cast<const float*>(sc.gate) + at + 4);
    } else {
      const uint4 v = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(sc.gate) + at);
      x = make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
      y = make_float4(__uint_as_float(v.z << 16), __uint_as_float(v.z & 0xffff0000u), __uint_as_float(v.w << 16), __uint_as_float(v.w & 0xffff0000u));
    }
    g[0] = sigmoid_of(x.x); g[1] = sigmoid_of(x.y); g[2] = sigmoid_of(x.z); g[3] = sigmoid_of(x.w);
    g[4] = sigmoid_of(y.x); g[5] = sigmoid_of(y.y); g[6] = sigmoid_of(y.z); g[7] = sigmoid_of(y.w);
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) g[e] = e < live ? gate_at(sc, row, c + e) : 0.f;
  }
}

// Four capped scores in log2 units: cap2 tanh(s to_cap) with tanh(x) = 1 - 2 / (1 + exp(2 x)); to2 = 2 log2(e) to_cap. One reciprocal serves
// the four (the exponents are held below 30, where the quotient is far below the last digit of one).
VE_DEVINL void cap2_of4(float* s, float to2, float cap2) {
  const float a = 1.f + ex2_approx(fminf(s[0] * to2, 30.f)), b = 1.f + ex2_approx(fminf(s[1] * to2, 30.f));
  const float c = 1.f + ex2_approx(fminf(s[2] * to2, 30.f)), d = 1.f + ex2_approx(fminf(s[3] * to2, 30.f));
  const float ab = a * b, cd = c * d, r = -2.f * cap2 * rcp_approx(ab * cd), rab = r * cd, rcd = r * ab;
  s[0] = fmaf(rab, b, cap2);
  s[1] = fmaf(rab, a, cap2);
  s[2] = fmaf(rcd, d, cap2);
  s[3] = fmaf(rcd, c, cap2);
}

template <int DQC, int DVC>
__global__ void __launch_bounds__(kGtThreads, 1) gqa_prefill_kernel(const GqaTc p, const __grid_constant__ CUtensorMap kmap,
                                                                    const __grid_constant__ CUtensorMap vmap) {
  constexpr int KS = GtStages<DQC, DVC>::K, VS = GtStages<DQC, DVC>::V, KB = DQC * 8192, VB = DVC * 8192, QC = kGtRows * 128, PB = kGtRows * 128, DV = DVC * 64;
  constexpr uint32_t TMEM_COLS = 512, O_COL = 256;       // S of stream t, buffer b at t * 128 + b * 64; O of stream t at 256 + t * DV
  const float NEG_INF = __int_as_float(0xff800000);
  grid_dep_wait();
  grid_dep_launch();
  extern __shared__ uint8_t gt_smem[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(gt_smem) + 1023) & ~(uintptr_t)1023);
  uint8_t* q_s = smem;                                   // [DQC][128 rows][128 B]
  uint8_t* k_s = q_s + DQC * QC;                         // [KS][DQC][64 keys][128 B]
  uint8_t* v_s = k_s + KS * KB;                          // [VS][DVC][64 keys][128 B]
  uint8_t* p_s = v_s + VS * VB;                       // [2 streams][2 terms][128 rows][128 B]
  __shared__ uint64_t kfull[KS], kempty[KS], vfull[VS], vempty[VS], s_full[2][2], p_full[2], pv_done[2];
  __shared__ uint32_t tmem_holder;
  __shared__ int s_fail;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int tile = gridDim.x - 1 - blockIdx.x, kvh = blockIdx.y, hpg = p.n.H / p.n.G;      // late tiles (many keys) first
  const int first = p.tile_first[tile], count = p.tile_count[tile], slot = p.rw.slot[first];
  if (slot < 0 || count <= 0) return;
  const int win = p.sc.window;
  const GqaPages pg(p.sc, p.rw.pos[first]);
  const int n = pg.count(p.rw.pos[first + count - 1]);                  // pages
  if (tid == 0) {
    for (int i = 0; i < KS; ++i) {
      mbar_init(&kfull[i], 1);
      mbar_init(&kempty[i], 1);
    }
    for (int i = 0; i < VS; ++i) {
      mbar_init(&vfull[i], 1);
      mbar_init(&vempty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i][0], 1);
      mbar_init(&s_full[i][1], 1);
      mbar_init(&p_full[i], 128);
      mbar_init(&pv_done[i], 1);
    }
    s_fail = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(&tmem_holder, TMEM_COLS);
    tmem_relinquish();
  }
  // a softmax thread owns one row of one stream: TMEM lane = 32 * (warp % 4) + lane, stream = (warp - 2) / 4
  const int r = (warp & 3) * 32 + lane, strm = warp >= 6 ? 1 : 0;
  const bool r_ok = warp >= 2 && r < count * hpg;
  const int r_tok = first + (r_ok ? r / hpg : 0), r_head = kvh * hpg + (r_ok ? r % hpg : 0), r_pos = p.rw.pos[r_tok];
  if (warp >= 2) {
    // the two streams' threads of a row share its 16-byte pieces of Q
    const __nv_bfloat16* src = p.q + ((long)r_tok * p.n.H + r_head) * p.n.kw;
#pragma unroll
    for (int i = 0; i < DQC * 4; ++i) {
      const int pc = 2 * i + strm, c = pc >> 3, col = c * 64 + (pc & 7) * 8;
      const uint4 v = r_ok && col < p.n.kw ? *reinterpret_cast<const uint4*>(src + col) : make_uint4(0u, 0u, 0u, 0u);
      *reinterpret_cast<uint4*>(q_s + c * QC + r * 128 + (((pc & 7) ^ (r & 7)) << 4)) = v;
    }
    fence_proxy_async_smem();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_holder;

  if (warp == 0) {
    // ------------------------------------------------------------------ page loads
    if (elect_one()) {
      prefetch_tmap(&kmap);
      prefetch_tmap(&vmap);
      for (int j = 0; j < n; ++j) {
        const int ks = j % KS, vs = j % VS, page = page_of(p.rw, slot, pg.of(j));
        if (j >= KS && !mbar_wait(&kempty[ks], ((j / KS) - 1) & 1)) {
          atomicExch(&s_fail, 1);
          break;
        }
        mbar_expect_tx(&kfull[ks], KB);
#pragma unroll
        for (int c = 0; c < DQC; ++c) tma_load_3d(k_s + ks * KB + c * 8192, &kmap, &kfull[ks], c * 64, kvh * kGPage, page);
        if (j >= VS && !mbar_wait(&vempty[vs], ((j / VS) - 1) & 1)) {
          atomicExch(&s_fail, 1);
          break;
        }
        mbar_expect_tx(&vfull[vs], VB);
#pragma unroll
        for (int c = 0; c < DVC; ++c) tma_load_3d(v_s + vs * VB + c * 8192, &vmap, &vfull[vs], c * 64, kvh * kGPage, page);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issue
    if (elect_one()) {
      constexpr uint32_t idesc_s = make_idesc_f16(1, 1, kGtRows, 64);
      constexpr uint32_t idesc_pv = make_idesc_f16(1, 1, kGtRows, DV) | (1u << 16);      // B (the values) is MN-major
      const uint32_t q_a = smem_u32(q_s), k_a = smem_u32(k_s), v_a = smem_u32(v_s), p_a = smem_u32(p_s);
      // page j belongs to stream j & 1 and is that stream's page j >> 1
      auto issue_s = [&](int j) {
        const int ks = j % KS, t = j & 1, b = (j >> 1) & 1;
        if (!mbar_wait(&kfull[ks], (j / KS) & 1)) return false;
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < DQC * 4; ++kk) {
          const int c = kk >> 2, off = (kk & 3) * 2;
          tc_mma_f16(tmem_base + t * 128 + b * 64, make_desc_sw128(q_a + c * QC) + off, make_desc_sw128(k_a + ks * KB + c * 8192) + off, idesc_s,
                     kk ? 1u : 0u);
        }
        tc_commit(&s_full[t][b]);
        tc_commit(&kempty[ks]);
        return true;
      };
      bool ok = issue_s(0);
      if (ok && n > 1) ok = issue_s(1);
      for (int j = 0; j < n && ok; ++j) {
        // the S buffer page j + 2 lands in was read by the softmax of page j - 2, which ended before its P arrived
        if (j + 2 < n) ok = issue_s(j + 2);
        if (!ok) break;
        const int t = j & 1, i = j >> 1, vs = j % VS;
        ok = mbar_wait(&vfull[vs], (j / VS) & 1) && mbar_wait(&p_full[t], i & 1);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int ks = 0; ks < 4; ++ks)
            tc_mma_f16(tmem_base + O_COL + t * DV, make_desc_sw128(p_a + (t * 2 + term) * PB) + ks * 2,
                       make_desc_sw128_mn(v_a + vs * VB + ks * 2048, 8192u, 1024u), idesc_pv, (i | ks | term) ? 1u : 0u);
        tc_commit(&pv_done[t]);
        tc_commit(&vempty[vs]);
      }
      if (!ok) atomicExch(&s_fail, 1);
    }
  } else {
    // ------------------------------------------------------------------ softmax and correction of one stream
    const uint32_t t_lane = tmem_base + ((uint32_t)((warp & 3) * 32) << 16);
    const uint32_t o_col = O_COL + strm * DV;
    const int n_mine = (n - strm + 1) >> 1;
    const bool capped = p.sc.cap > 0.f;
    const float cap2 = p.sc.cap * kLog2e, to2 = capped ? 2.f * kLog2e * p.sc.scale / p.sc.cap : 0.f;
    const float scale2 = capped ? 1.f : p.sc.scale * kLog2e;           // of what is in sv behind the cap
    const float* tab = p.sc.bias + (long)r_head * p.sc.L;
    const int L1 = p.sc.bias ? p.sc.L - 1 : 0;
    const float far = p.sc.bias ? tab[L1] * kLog2e : 0.f;
    float m_ref = NEG_INF, l0 = 0.f, l1 = 0.f;
    bool ok = true;
    uint8_t* prow = p_s + strm * 2 * PB + r * 128;
    for (int i = 0; i < n_mine; ++i) {
      const int b = i & 1, key0 = pg.of(2 * i + strm) * 64;
      ok = __all_sync(0xffffffffu, mbar_wait(&s_full[strm][b], (i >> 1) & 1));
      if (!ok) break;
      tc_fence_after();
      float sv[64];
      tmem_ld32(t_lane + strm * 128 + b * 64, reinterpret_cast<uint32_t*>(sv));
      tmem_ld32(t_lane + strm * 128 + b * 64 + 32, reinterpret_cast<uint32_t*>(sv) + 32);
      tmem_ld_wait();
      if (capped) {
#pragma unroll
        for (int e = 0; e < 64; e += 4) cap2_of4(sv + e, to2, cap2);
      }
      // far pages: the scores stay as they are and one addend per row stands for the bias; near pages: scaled, bias by distance
      const bool near = p.sc.bias && __any_sync(0xffffffffu, r_pos - key0 - 63 < L1);
      if (near) {
#pragma unroll
        for (int e = 0; e < 64; ++e) sv[e] = fmaf(sv[e], scale2, tab[min(max(r_pos - key0 - e, 0), L1)] * kLog2e);
      }
      const float mul = near ? 1.f : scale2, add = near ? 0.f : far;
      if (!r_ok || key0 + 63 > r_pos || r_pos - key0 >= win) {
#pragma unroll
        for (int e = 0; e < 64; ++e) sv[e] = r_ok && sees(p.sc, r_pos - key0 - e, key0 + e) ? sv[e] : NEG_INF;
      }
      float mx0 = sv[0], mx1 = sv[1], mx2 = sv[2], mx3 = sv[3];
#pragma unroll
      for (int e = 4; e < 64; e += 4) {
        mx0 = fmaxf(mx0, sv[e]);
        mx1 = fmaxf(mx1, sv[e + 1]);
        mx2 = fmaxf(mx2, sv[e + 2]);
        mx3 = fmaxf(mx3, sv[e + 3]);
      }
      const float mx = fmaf(fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)), mul, add);          // the scale is positive
      const bool grow = mx > m_ref + kGtLazyLog2;
      float alpha = 1.f;
      if (grow) {
        alpha = ex2_approx(m_ref - mx);                  // 0 for the first keys a row sees
        m_ref = mx;
      }
      const bool fix = i > 0 && __any_sync(0xffffffffu, grow);
      if (fix) {                                         // the stream's previous PV is the last writer of O
        ok = __all_sync(0xffffffffu, mbar_wait(&pv_done[strm], (i - 1) & 1));
        if (!ok) break;
        tc_fence_after();
#pragma unroll 1
        for (int c0 = 0; c0 < DV; c0 += 32) {
          uint32_t ov[32];
          tmem_ld32(t_lane + o_col + c0, ov);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 32; ++e) ov[e] = __float_as_uint(__uint_as_float(ov[e]) * alpha);
          tmem_st32(t_lane + o_col + c0, ov);
        }
        tmem_st_wait();
      }
      l0 *= alpha;
      l1 *= alpha;
      const float neg_m = add - (m_ref == NEG_INF ? 0.f : m_ref);
      uint32_t w[32], x[32];                             // leading terms and remainders
#pragma unroll
      for (int e = 0; e < 32; ++e) {
        const float p0 = ex2_approx(fmaf(sv[2 * e], mul, neg_m)), p1 = ex2_approx(fmaf(sv[2 * e + 1], mul, neg_m));
        l0 += p0;
        l1 += p1;
        w[e] = gq_pack(p0, p1);
        x[e] = gq_pack(p0 - __uint_as_float(w[e] << 16), p1 - __uint_as_float(w[e] & 0xffff0000u));
      }
      if (i > 0 && !fix) {
        ok = __all_sync(0xffffffffu, mbar_wait(&pv_done[strm], (i - 1) & 1));
        if (!ok) break;
      }
#pragma unroll
      for (int ch = 0; ch < 8; ++ch) {
        const int at = (ch ^ (r & 7)) << 4;
        *reinterpret_cast<uint4*>(prow + at) = make_uint4(w[4 * ch], w[4 * ch + 1], w[4 * ch + 2], w[4 * ch + 3]);
        *reinterpret_cast<uint4*>(prow + PB + at) = make_uint4(x[4 * ch], x[4 * ch + 1], x[4 * ch + 2], x[4 * ch + 3]);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(&p_full[strm]);
    }
    if (n_mine > 0) ok = __all_sync(0xffffffffu, ok && mbar_wait(&pv_done[strm], (n_mine - 1) & 1));
    if (!ok) atomicExch(&s_fail, 1);
    // the stream's P buffer is free now (its last PV has completed): it carries (reference, sum) to the merge
    reinterpret_cast<float*>(p_s + strm * 2 * PB)[r] = m_ref;
    reinterpret_cast<float*>(p_s + strm * 2 * PB)[kGtRows + r] = l0 + l1;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp >= 2 && !s_fail) {
    // ------------------------------------------------------------------ merge of the two streams and the sink, output
    const uint32_t t_lane = tmem_base + ((uint32_t)((warp & 3) * 32) << 16);
    const float* ml0 = reinterpret_cast<const float*>(p_s);
    const float* ml1 = reinterpret_cast<const float*>(p_s + 2 * PB);
    const float snk = p.sc.sink ? p.sc.sink[r_head] * kLog2e : NEG_INF;
    const float m0 = ml0[r], m1 = ml1[r], m = fmaxf(snk, fmaxf(m0, m1));
    const float a0 = m0 == NEG_INF ? 0.f : ex2_approx(m0 - m), a1 = (m1 == NEG_INF || n < 2) ? 0.f : ex2_approx(m1 - m);
    const float l = ml0[kGtRows + r] * a0 + (n < 2 ? 0.f : ml1[kGtRows + r] * a1) + (p.sc.sink ? ex2_approx(snk - m) : 0.f);
    const float inv = l > 0.f ? p.sc.out_scale / l : 0.f, f0 = a0 * inv, f1 = a1 * inv;
    __nv_bfloat16* orow = p.out + (long)r_tok * p.ldo + (long)r_head * p.n.dv;
#pragma unroll 1
    for (int c0 = strm * DVC * 32; c0 < (strm + 1) * DVC * 32; c0 += 32) {
      uint32_t ov[32], ow[32];
      tmem_ld32(t_lane + O_COL + c0, ov);
      if (n > 1) tmem_ld32(t_lane + O_COL + DV + c0, ow);     // a one-page sequence never wrote the second accumulator
      tmem_ld_wait();
      if (r_ok) {
#pragma unroll
        for (int q4 = 0; q4 < 4; ++q4) {
          const int col = c0 + q4 * 8;
          if (col >= p.n.dv) continue;
          uint32_t w[4];
          float gt[8];
          gate8(p.sc, r_tok, r_head * p.n.dv + col, p.n.dv - col, gt);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float a = __uint_as_float(ov[q4 * 8 + 2 * e]) * f0, c = __uint_as_float(ov[q4 * 8 + 2 * e + 1]) * f0;
            if (n > 1) {
              a = fmaf(__uint_as_float(ow[q4 * 8 + 2 * e]), f1, a);
              c = fmaf(__uint_as_float(ow[q4 * 8 + 2 * e + 1]), f1, c);
            }
            if (p.sc.back) {                             // (only pairs that exist: the last columns of eight may not)
              const int m = (col >> 1) + e;
              const float2 z = m < p.sc.bpairs ? p.sc.back[(long)r_tok * p.sc.bpairs + m] : make_float2(0.f, 0.f);
              const float x = fmaf(a, z.x, c * z.y);
              c = fmaf(c, z.x, -(a * z.y));
              a = x;
            }
            w[e] = gq_pack(a * gt[2 * e], c * gt[2 * e + 1]);
          }
          if (p.vec) *reinterpret_cast<uint4*>(orow + col) = make_uint4(w[0], w[1], w[2], w[3]);
          else
#pragma unroll
            for (int e = 0; e < 8; ++e)
              if (col + e < p.n.dv) orow[col + e] = __ushort_as_bfloat16((unsigned short)(w[e >> 1] >> (16 * (e & 1))));
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
  if (tid == 0 && s_fail && p.status) atomicExch(p.status, (int)kErrMbarTimeout);
}

template <int DQC, int DVC>
static int launch_gqa_tc(const GqaTc& p, const CUtensorMap& km, const CUtensorMap& vm, int ntiles, cudaStream_t st) {
  constexpr int smem = DQC * kGtRows * 128 + GtStages<DQC, DVC>::K * DQC * 8192 + GtStages<DQC, DVC>::V * DVC * 8192 + 4 * kGtRows * 128 + 1024;
  static_assert(smem <= 227 * 1024 - 512, "shared memory budget");
  static bool attr = false;
  if (!attr) {
    const cudaError_t e = cudaFuncSetAttribute(gqa_prefill_kernel<DQC, DVC>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
    attr = true;
  }
  launch_pdl(gqa_prefill_kernel<DQC, DVC>, dim3(ntiles, p.n.G), dim3(kGtThreads), smem, st, p, km, vm);
  return (int)cudaGetLastError();
}

}  // namespace ve
