// Latent attention of prompt rows on the fifth-generation tensor cores (tcgen05, accumulators in TMEM). Included by latent.cu.
//
// One CTA = 128 query rows of one sequence and head against 64-key tiles of its expanded keys and values. The structure is that of
// attention_tc.cuh (two streams of alternating key tiles, each with its own S buffers, softmax warps, running reference and O
// accumulator; lazy moves of the reference; merge in the epilogue) with these differences:
//   * query and key are DQC chunks of 64 columns (plain part, then rotated part; pad columns of the query are zero), the key's
//     rotated part comes from the cached rows and is shared by the heads; values are DVC chunks;
//   * the softmax weights enter the second product as two bf16 terms (value and remainder), so they keep 32-bit quality;
//   * keys and values have rings and loaders of their own (a key tile is free as soon as its scores are done, and its successor is not
//     requested behind values that wait for their weights): warps 0 and 10;
//   * with a sliding window the key tiles in front of the first row's window are not visited.
// Every wait is bounded; on expiry the CTA records a status code, skips its stores and frees its TMEM.
#pragma once

namespace ve {

struct LatentTc {
  LatentDims n;
  const __nv_bfloat16* q; long ldq;        // [rows][H (d + rot)], rotated
  const int* pos;
  const int* tile_first; const int* tile_count; const int* tile_base;
  const int* tile_key0;                    // position of the key row tile_base
  int window;
  __nv_bfloat16* out; long ldo;
  float scale_log2;
  int uc;                                  // chunks of the plain part
  int* status;
};

constexpr int kLtRows = 128, kLtThreads = 352, kLtKs = 3, kLtVs = 2;
constexpr float kLtLazyLog2 = 8.f;

template <int DQC, int DVC>
__global__ void __launch_bounds__(kLtThreads, 1) latent_prefill_tc_kernel(const LatentTc p, const __grid_constant__ CUtensorMap upmap,
                                                                          const __grid_constant__ CUtensorMap rotmap) {
  constexpr int KB = DQC * 8192, VB = DVC * 8192, QC = kLtRows * 128, PB = kLtRows * 128, DV = DVC * 64;
  constexpr uint32_t TMEM_COLS = 512, O_COL = 256;       // S of stream t, buffer b at t * 128 + b * 64; O of stream t at 256 + t * DV
  const float NEG_INF = __int_as_float(0xff800000);
  grid_dep_wait();
  grid_dep_launch();
  extern __shared__ uint8_t lt_smem[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lt_smem) + 1023) & ~(uintptr_t)1023);
  uint8_t* q_s = smem;                                   // [DQC][128 rows][128 B]
  uint8_t* k_s = q_s + DQC * QC;                         // [kLtKs][DQC][64 keys][128 B]
  uint8_t* v_s = k_s + kLtKs * KB;                       // [kLtVs][DVC][64 keys][128 B]
  uint8_t* p_s = v_s + kLtVs * VB;                       // [2 streams][2 terms][128 rows][128 B]
  __shared__ uint64_t kfull[kLtKs], kempty[kLtKs], vfull[kLtVs], vempty[kLtVs], s_full[2][2], p_full[2], pv_done[2];
  __shared__ uint32_t tmem_holder;
  __shared__ int s_fail;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int tile = gridDim.x - 1 - blockIdx.x, h = blockIdx.y;          // late tiles (many keys) first
  const int first = p.tile_first[tile], count = p.tile_count[tile], win = p.window;
  const int skip = max(0, p.pos[first] - win + 1 - p.tile_key0[tile]) / kLPage * kLPage;      // key rows that no row of the tile sees
  const int kbase = p.tile_base[tile] + skip, kpos = p.tile_key0[tile] + skip;                // first key row and its position
  const int n = (p.pos[first + count - 1] - kpos) / kLPage + 1;         // key tiles
  if (tid == 0) {
    for (int i = 0; i < kLtKs; ++i) {
      mbar_init(&kfull[i], 1);
      mbar_init(&kempty[i], 1);
    }
    for (int i = 0; i < kLtVs; ++i) {
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
  const bool soft = warp >= 2 && warp < 10, r_ok = soft && r < count;
  const int r_tok = first + (r_ok ? r : 0), r_pos = p.pos[r_tok];
  if (soft) {
    // the two streams' threads of a row share its 16-byte pieces of Q
    const __nv_bfloat16* src = p.q + (long)r_tok * p.ldq + (long)h * (p.n.d + p.n.rot);
#pragma unroll
    for (int i = 0; i < DQC * 4; ++i) {
      const int pc = 2 * i + strm, c = pc >> 3, w = (pc & 7) * 8;
      const bool plain = c < p.uc;
      const int col = plain ? c * 64 + w : p.n.d + (c - p.uc) * 64 + w;
      const bool in = r_ok && col < (plain ? p.n.d : p.n.d + p.n.rot);
      const uint4 v = in ? *reinterpret_cast<const uint4*>(src + col) : make_uint4(0u, 0u, 0u, 0u);
      *reinterpret_cast<uint4*>(q_s + c * QC + r * 128 + (((pc & 7) ^ (r & 7)) << 4)) = v;
    }
    fence_proxy_async_smem();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_holder;

  if (warp == 0) {
    // ------------------------------------------------------------------ key loads
    if (elect_one()) {
      prefetch_tmap(&upmap);
      prefetch_tmap(&rotmap);
      for (int j = 0; j < n; ++j) {
        const int ks = j % kLtKs, row = kbase + j * 64;
        if (j >= kLtKs && !mbar_wait(&kempty[ks], ((j / kLtKs) - 1) & 1)) {
          atomicExch(&s_fail, 1);
          break;
        }
        mbar_expect_tx(&kfull[ks], KB);
#pragma unroll
        for (int c = 0; c < DQC; ++c) {
          if (c < p.uc) tma_load_2d(k_s + ks * KB + c * 8192, &upmap, &kfull[ks], h * p.n.d + c * 64, row);
          else tma_load_2d(k_s + ks * KB + c * 8192, &rotmap, &kfull[ks], p.n.rot0 + (c - p.uc) * 64, row);
        }
      }
    }
  } else if (warp == 10) {
    // ------------------------------------------------------------------ value loads
    if (elect_one()) {
      for (int j = 0; j < n; ++j) {
        const int vs = j % kLtVs, row = kbase + j * 64;
        if (j >= kLtVs && !mbar_wait(&vempty[vs], ((j / kLtVs) - 1) & 1)) {
          atomicExch(&s_fail, 1);
          break;
        }
        mbar_expect_tx(&vfull[vs], VB);
#pragma unroll
        for (int c = 0; c < DVC; ++c)
          tma_load_2d(v_s + vs * VB + c * 8192, &upmap, &vfull[vs], p.n.H * p.n.d + h * p.n.dv + c * 64, row);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issue
    if (elect_one()) {
      constexpr uint32_t idesc_s = make_idesc_f16(1, 1, kLtRows, 64);
      constexpr uint32_t idesc_pv = make_idesc_f16(1, 1, kLtRows, DV) | (1u << 16);      // B (the values) is MN-major
      const uint32_t q_a = smem_u32(q_s), k_a = smem_u32(k_s), v_a = smem_u32(v_s), p_a = smem_u32(p_s);
      // key tile j belongs to stream j & 1 and is that stream's tile j >> 1
      auto issue_s = [&](int j) {
        const int ks = j % kLtKs, t = j & 1, b = (j >> 1) & 1;
        if (!mbar_wait(&kfull[ks], (j / kLtKs) & 1)) return false;
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
        // the S buffer tile j + 2 lands in was read by the softmax of tile j - 2, which ended before its P arrived
        if (j + 2 < n) ok = issue_s(j + 2);
        if (!ok) break;
        const int t = j & 1, i = j >> 1, vs = j % kLtVs;
        ok = mbar_wait(&vfull[vs], (j / kLtVs) & 1) && mbar_wait(&p_full[t], i & 1);
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
    float m_ref = NEG_INF, l0 = 0.f, l1 = 0.f;
    bool ok = true;
    uint8_t* prow = p_s + strm * 2 * PB + r * 128;
    for (int i = 0; i < n_mine; ++i) {
      const int b = i & 1, key0 = kpos + (2 * i + strm) * 64;
      ok = __all_sync(0xffffffffu, mbar_wait(&s_full[strm][b], (i >> 1) & 1));
      if (!ok) break;
      tc_fence_after();
      float sv[64];
      tmem_ld32(t_lane + strm * 128 + b * 64, reinterpret_cast<uint32_t*>(sv));
      tmem_ld32(t_lane + strm * 128 + b * 64 + 32, reinterpret_cast<uint32_t*>(sv) + 32);
      tmem_ld_wait();
      if (!r_ok || key0 + 63 > r_pos || r_pos - key0 >= win) {
#pragma unroll
        for (int e = 0; e < 64; ++e) sv[e] = r_ok && (unsigned)(r_pos - key0 - e) < (unsigned)win ? sv[e] : NEG_INF;
      }
      float mx0 = sv[0], mx1 = sv[1], mx2 = sv[2], mx3 = sv[3];
#pragma unroll
      for (int e = 4; e < 64; e += 4) {
        mx0 = fmaxf(mx0, sv[e]);
        mx1 = fmaxf(mx1, sv[e + 1]);
        mx2 = fmaxf(mx2, sv[e + 2]);
        mx3 = fmaxf(mx3, sv[e + 3]);
      }
      const float mx = fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)) * p.scale_log2;     // the scale is positive
      const bool grow = mx > m_ref + kLtLazyLog2;
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
      const float neg_m = m_ref == NEG_INF ? 0.f : -m_ref;
      uint32_t w[32], x[32];                             // leading terms and remainders
#pragma unroll
      for (int e = 0; e < 32; ++e) {
        const float p0 = ex2_approx(fmaf(sv[2 * e], p.scale_log2, neg_m)), p1 = ex2_approx(fmaf(sv[2 * e + 1], p.scale_log2, neg_m));
        l0 += p0;
        l1 += p1;
        w[e] = lp_pack(p0, p1);
        x[e] = lp_pack(p0 - __uint_as_float(w[e] << 16), p1 - __uint_as_float(w[e] & 0xffff0000u));
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
    reinterpret_cast<float*>(p_s + strm * 2 * PB)[kLtRows + r] = l0 + l1;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (soft && !s_fail) {
    // ------------------------------------------------------------------ merge of the two streams and output
    const uint32_t t_lane = tmem_base + ((uint32_t)((warp & 3) * 32) << 16);
    const float* ml0 = reinterpret_cast<const float*>(p_s);
    const float* ml1 = reinterpret_cast<const float*>(p_s + 2 * PB);
    const float m0 = ml0[r], m1 = ml1[r], m = fmaxf(m0, m1);
    const float a0 = m == NEG_INF ? 0.f : ex2_approx(m0 - m), a1 = (m == NEG_INF || n < 2) ? 0.f : ex2_approx(m1 - m);
    const float l = ml0[kLtRows + r] * a0 + (n < 2 ? 0.f : ml1[kLtRows + r] * a1);
    const float inv = l > 0.f ? 1.f / l : 0.f, f0 = a0 * inv, f1 = a1 * inv;
    __nv_bfloat16* orow = p.out + (long)r_tok * p.ldo + (long)h * p.n.dv;
#pragma unroll 1
    for (int c0 = strm * DVC * 32; c0 < (strm + 1) * DVC * 32; c0 += 32) {
      uint32_t ov[32], ow[32];
      tmem_ld32(t_lane + O_COL + c0, ov);
      if (n > 1) tmem_ld32(t_lane + O_COL + DV + c0, ow);     // a one-tile sequence never wrote the second accumulator
      tmem_ld_wait();
      if (r_ok) {
#pragma unroll
        for (int q4 = 0; q4 < 4; ++q4) {
          if (c0 + q4 * 8 >= p.n.dv) continue;
          uint32_t w[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float a = __uint_as_float(ov[q4 * 8 + 2 * e]) * f0, c = __uint_as_float(ov[q4 * 8 + 2 * e + 1]) * f0;
            if (n > 1) {
              a = fmaf(__uint_as_float(ow[q4 * 8 + 2 * e]), f1, a);
              c = fmaf(__uint_as_float(ow[q4 * 8 + 2 * e + 1]), f1, c);
            }
            w[e] = lp_pack(a, c);
          }
          *reinterpret_cast<uint4*>(orow + c0 + q4 * 8) = make_uint4(w[0], w[1], w[2], w[3]);
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
static int launch_latent_tc(const LatentTc& p, const CUtensorMap& up, const CUtensorMap& rot, int ntiles, cudaStream_t st) {
  constexpr int smem = DQC * kLtRows * 128 + kLtKs * DQC * 8192 + kLtVs * DVC * 8192 + 4 * kLtRows * 128 + 1024;
  static_assert(smem <= 227 * 1024, "shared memory budget");
  static bool attr = false;
  if (!attr) {
    cudaError_t e = cudaFuncSetAttribute(latent_prefill_tc_kernel<DQC, DVC>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
    attr = true;
  }
  launch_pdl(latent_prefill_tc_kernel<DQC, DVC>, dim3(ntiles, p.n.H), dim3(kLtThreads), smem, st, p, up, rot);
  return (int)cudaGetLastError();
}

}  // namespace ve
