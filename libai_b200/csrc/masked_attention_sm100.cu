// Prompt attention under a position mask for sm_100a on tcgen05 / TMEM / TMA (bf16): grouped query heads of D channels and values of V
// (multiples of 16, at most 128), ragged sequences that may continue cached rows, a causal mask that reaches back to position 0, to the
// start of the query's chunk or over a sliding window, an optional query temperature by position and an optional sigmoid output gate.
//
// One CTA per (head, tile of 128 consecutive queries of one sequence), 320 threads:
//   warp 0        TMA producer : the query tile once (64-channel chunks), then key and value tiles of 128 rows from the row matrices, both
//                                double buffered; only tiles with a row that some query of the tile sees are visited
//   warp 1        MMA issuer   : S = Q K^T into TMEM, O += P V with P read from TMEM
//   warps 2..9    softmax      : two threads per query row: online softmax, P (bf16) to TMEM, the output kept in TMEM and rescaled only
//                                when the running maximum grows by more than 2^8
// Values are padded to VP = 64 or 128 columns: the columns beyond V hold the next head's values (or zeros) and are never stored.
// Every wait on an mbarrier is bounded: when one runs out, the CTA stops issuing copies and products, runs its (finite) loops to
// the end without waiting, lets the copies in flight land, frees its TMEM and reports through `err`.
#include "attention_tc.cuh"

namespace lb {

constexpr int MTC_BM = 128, MTC_BN = 128, MTC_THREADS = 320;

template <int DC, int VP>    // DC: 64-channel chunks of a query / key head; VP: padded value channels
struct MtcCfg {
  static constexpr int CHUNK = 128 * 128;                               // 128 rows x 64 bf16
  static constexpr int Q_BYTES = DC * CHUNK, K_BYTES = Q_BYTES, V_BYTES = (VP / 64) * CHUNK;
  static constexpr int XCHG_BYTES = 2 * 2 * 128 * 4;                    // row maxima exchanged between the two halves: [parity][half][row]
  static constexpr int SMEM_BYTES = Q_BYTES + 2 * K_BYTES + 2 * V_BYTES + XCHG_BYTES + 1024 + 256;
  static constexpr uint32_t TMEM_COLS = VP == 64 ? 256 : 512;
  static constexpr uint32_t S_COL = 0, O_COL = 128, P_COL = 128 + VP;
};

struct MtcParams {
  __nv_bfloat16* y;
  long ldy;
  const __nv_bfloat16* gate;  // [tokens, H] or — gate_wide — [tokens, H*V], or null
  long ldg;
  const int *qt_seq, *qt_start, *seq_off, *past, *ext_off, *nsink, *cstart;
  int H, G, D, V, window, chunk, gate_wide;
  float scale_log2, out_scale, temp_coef, temp_every;
  int* err;                   // mapped host word, set when a wait ran out
};

LB_DEVICE int mtc_floor(int p, int window, int chunk) {
  return chunk > 0 ? (p / chunk) * chunk : (window > 0 ? max(0, p - window + 1) : 0);
}
LB_DEVICE float mtc_sigmoid(float x) { return 1.0f / (1.0f + __expf(-x)); }

template <int DC, int VP>
__global__ void __launch_bounds__(MTC_THREADS, VP == 64 && DC == 1 ? 2 : 1)
masked_attention_tc_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                           const __grid_constant__ CUtensorMap tmap_v, MtcParams p) {
  using Cfg = MtcCfg<DC, VP>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + Cfg::Q_BYTES;
  uint8_t* sV = sK + 2 * Cfg::K_BYTES;
  float* sXchg = reinterpret_cast<float*>(sV + 2 * Cfg::V_BYTES);
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + 2 * Cfg::V_BYTES + Cfg::XCHG_BYTES);
  uint64_t *q_full = bars, *k_full = bars + 2, *k_empty = bars + 4, *v_full = bars + 6, *v_empty = bars + 8;
  uint64_t *s_full = bars + 10, *p_full = bars + 11, *o_full = bars + 12, *s_free = bars + 13;
  uint32_t* tmem_ptr_smem = reinterpret_cast<uint32_t*>(bars + 14);
  volatile int* stop = reinterpret_cast<volatile int*>(bars + 15);

  const int warp_idx = threadIdx.x / 32, lane = threadIdx.x % 32;
  const int head = blockIdx.x, g = head / (p.H / p.G), b = p.qt_seq[blockIdx.y], t0 = p.qt_start[blockIdx.y];
  const int tok0 = p.seq_off[b] + t0, nq = min(MTC_BM, p.seq_off[b + 1] - tok0);
  const int pos0 = p.past[b] + t0;
  const int key0 = mtc_floor(pos0, p.window, p.chunk);                  // first position that a query of the tile sees
  const int row0 = p.ext_off[b] + p.nsink[b] + key0 - p.cstart[b];                   // its row
  const int nkv = (pos0 + nq - 1 - key0) / MTC_BN + 1;                  // key tiles up to the tile's last query

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmap_q);
    tma_prefetch_desc(&tmap_k);
    tma_prefetch_desc(&tmap_v);
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) { mbar_init(&k_full[i], 1); mbar_init(&k_empty[i], 1); mbar_init(&v_full[i], 1); mbar_init(&v_empty[i], 1); }
    mbar_init(s_full, 1);
    mbar_init(p_full, 8);
    mbar_init(o_full, 1);
    mbar_init(s_free, 8);
    *stop = 0;
    fence_barrier_init();
    fence_proxy_async();
  }
  if (warp_idx == 1) tmem_alloc<Cfg::TMEM_COLS>(tmem_ptr_smem);
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_ptr_smem;

  if (warp_idx == 0) {
    if (elect_one()) {
      mbar_arrive_expect_tx(q_full, Cfg::Q_BYTES);
#pragma unroll
      for (int c = 0; c < DC; ++c) tma_load_3d(sQ + c * Cfg::CHUNK, &tmap_q, q_full, c * 64, head, tok0);
      for (int j = 0; j < nkv; ++j) {
        const int s = j & 1, row = row0 + j * MTC_BN;
        const uint32_t par = ((j >> 1) & 1) ^ 1;
        if (tc_wait(&k_empty[s], par, stop)) {
          mbar_arrive_expect_tx(&k_full[s], Cfg::K_BYTES);
#pragma unroll
          for (int c = 0; c < DC; ++c) tma_load_2d(sK + s * Cfg::K_BYTES + c * Cfg::CHUNK, &tmap_k, &k_full[s], g * p.D + c * 64, row);
        }
        if (tc_wait(&v_empty[s], par, stop)) {
          mbar_arrive_expect_tx(&v_full[s], Cfg::V_BYTES);
#pragma unroll
          for (int c = 0; c < VP / 64; ++c) tma_load_2d(sV + s * Cfg::V_BYTES + c * Cfg::CHUNK, &tmap_v, &v_full[s], g * p.V + c * 64, row);
        }
      }
    }
    __syncwarp();
  } else if (warp_idx == 1) {
    constexpr uint32_t idesc_qk = make_idesc_bf16(MTC_BM, MTC_BN, false, false);
    constexpr uint32_t idesc_pv = make_idesc_bf16(MTC_BM, VP, false, true);
    const uint32_t q_addr = smem_u32(sQ);
    const int ksteps = p.D / 16;
    bool ok = __all_sync(0xffffffffu, tc_wait(q_full, 0, stop));
    // S(j + 1) is issued as soon as the softmax warps have read S(j) for the last time, ahead of P(j) V(j)
    auto issue_qk = [&](int j) {
      const int s = j & 1;
      ok = __all_sync(0xffffffffu, ok && tc_wait(&k_full[s], (j >> 1) & 1, stop));
      if (j > 0) ok = __all_sync(0xffffffffu, ok && tc_wait(s_free, (j - 1) & 1, stop));
      tc_fence_after_sync();
      if (ok && elect_one()) {
        const uint32_t k_addr = smem_u32(sK + s * Cfg::K_BYTES);
#pragma unroll
        for (int kk = 0; kk < DC * 4; ++kk) {
          if (kk < ksteps) {
            const uint32_t off = (kk / 4) * Cfg::CHUNK + (kk % 4) * 32;
            umma_f16_ss(tmem_base + Cfg::S_COL, make_smem_desc_sw128(q_addr + off, 0, 1024), make_smem_desc_sw128(k_addr + off, 0, 1024),
                        idesc_qk, kk > 0 ? 1u : 0u);
          }
        }
        umma_commit(s_full);
        umma_commit(&k_empty[s]);
      }
      __syncwarp();
    };
    issue_qk(0);
    for (int j = 0; j < nkv; ++j) {
      const int s = j & 1;
      if (j + 1 < nkv) issue_qk(j + 1);
      ok = __all_sync(0xffffffffu, ok && tc_wait(p_full, j & 1, stop));
      ok = __all_sync(0xffffffffu, ok && tc_wait(&v_full[s], (j >> 1) & 1, stop));
      tc_fence_after_sync();
      if (ok && elect_one()) {
        const uint32_t v_addr = smem_u32(sV + s * Cfg::V_BYTES);
#pragma unroll
        for (int kk = 0; kk < MTC_BN / 16; ++kk)
          umma_f16_ts(tmem_base + Cfg::O_COL, tmem_base + Cfg::P_COL + kk * 8,
                      make_smem_desc_sw128(v_addr + kk * (16 * 128), MTC_BN * 128, 1024), idesc_pv, (j > 0 || kk > 0) ? 1u : 0u);
        umma_commit(o_full);
        umma_commit(&v_empty[s]);
      }
      __syncwarp();
    }
  } else {
    const int quad = warp_idx % 4, half = (warp_idx - 2) / 4;           // this warp's 64 of the 128 key columns
    const int r = quad * 32 + lane;                                     // query row of this thread (shared with the other half's thread)
    const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t s_addr = tmem_base + lane_off + Cfg::S_COL + half * 64;
    const uint32_t p_addr = tmem_base + lane_off + Cfg::P_COL + half * 32;
    const uint32_t o_addr = tmem_base + lane_off + Cfg::O_COL + half * (VP / 2);
    const float scale = p.scale_log2 * (p.temp_every > 0.f ? 1.f + p.temp_coef * logf(floorf(static_cast<float>(pos0 + r + 1) / p.temp_every) + 1.f) : 1.f);
    float m_run = -INFINITY, l_run = 0.f;                               // log2 domain; l_run: the sum over this half's columns
    const int key_lo = mtc_floor(pos0 + r, p.window, p.chunk), key_lim = pos0 + r + 1;      // this row sees the positions [key_lo, key_lim)
    const int last_lo = mtc_floor(pos0 + MTC_BM - 1, p.window, p.chunk);
    for (int j = 0; j < nkv; ++j) {
      tc_wait(s_full, j & 1, stop);
      __syncwarp();
      tc_fence_after_sync();
      const int kt = key0 + j * MTC_BN, k0 = kt + half * 64;
      const bool need_mask = kt + MTC_BN > pos0 + 1 || kt < last_lo;    // some row of the tile does not see the whole key tile
      float mx = -INFINITY;
      auto pass1 = [&](auto mask_tag) {
        constexpr bool MASK = decltype(mask_tag)::value;
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          uint32_t t[32];
          tmem_ld_32x32b_x32(s_addr + c * 32, t);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            float x = __uint_as_float(t[i]);
            if constexpr (MASK) x = (k0 + c * 32 + i < key_lim && k0 + c * 32 + i >= key_lo) ? x : -INFINITY;
            mx = fmaxf(mx, x);
          }
        }
      };
      if (need_mask) pass1(std::true_type{}); else pass1(std::false_type{});
      float* xch = sXchg + (j & 1) * 256;
      xch[half * 128 + r] = mx;
      tc_pair_sync(quad);
      mx = fmaxf(mx, xch[(half ^ 1) * 128 + r]);
      const float m_cand = fmaxf(m_run, mx * scale);
      const bool bump = (m_cand - m_run > 8.0f) || (m_run == -INFINITY && m_cand != -INFINITY);
      float alpha = 1.0f;
      if (bump) { alpha = fast_exp2(m_run - m_cand); m_run = m_cand; }  // 0 on the first tile with a visible key
      const bool bump_any = __any_sync(0xffffffffu, bump && j > 0);
      const float m_use = m_run == -INFINITY ? 0.f : m_run;
      float rowsum = 0.f;
      auto pass2 = [&](auto mask_tag) {
        constexpr bool MASK = decltype(mask_tag)::value;
        float rs0 = 0.f, rs1 = 0.f;
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          uint32_t t[32];
          tmem_ld_32x32b_x32(s_addr + c * 32, t);
          tmem_ld_wait();
          if (c == 1) {                                                 // S(j) has been read for the last time
            tc_fence_before_sync();
            __syncwarp();
            if (lane == 0) mbar_arrive(s_free);
          }
          uint32_t packed[16];
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            float x0 = fast_exp2(__uint_as_float(t[i]) * scale - m_use), x1 = fast_exp2(__uint_as_float(t[i + 1]) * scale - m_use);
            if constexpr (MASK) {
              const int kidx = k0 + c * 32 + i;
              x0 = (kidx < key_lim && kidx >= key_lo) ? x0 : 0.f;
              x1 = (kidx + 1 < key_lim && kidx + 1 >= key_lo) ? x1 : 0.f;
            }
            rs0 += x0;
            rs1 += x1;
            packed[i / 2] = pack_bf16(x0, x1);
          }
          tmem_st_32x32b_x16(p_addr + c * 16, packed);
        }
        rowsum = rs0 + rs1;
      };
      // P(j) overwrites the columns that P(j - 1) V(j - 1) reads
      if (j > 0) { tc_wait(o_full, (j - 1) & 1, stop); __syncwarp(); tc_fence_after_sync(); }
      if (need_mask) pass2(std::true_type{}); else pass2(std::false_type{});
      l_run = l_run * alpha + rowsum;
      if (bump_any) {                                                   // rare: P(j - 1) V(j - 1) has retired, rescale this half's columns
#pragma unroll
        for (int c = 0; c < VP / 64; ++c) {
          uint32_t t[32];
          tmem_ld_32x32b_x32(o_addr + c * 32, t);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) t[i] = __float_as_uint(__uint_as_float(t[i]) * alpha);
          tmem_st_32x32b_x32(o_addr + c * 32, t);
        }
      }
      tmem_st_wait();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    float* xch = sXchg + (nkv & 1) * 256;
    xch[half * 128 + r] = l_run;
    tc_pair_sync(quad);
    l_run += xch[(half ^ 1) * 128 + r];
    tc_wait(o_full, (nkv - 1) & 1, stop);
    __syncwarp();
    tc_fence_after_sync();
    float inv = l_run > 0.f ? p.out_scale / l_run : 0.f;
    const long tok = static_cast<long>(tok0) + r;
    const __nv_bfloat16* grow = nullptr;                                // this row's gate logits, one per channel
    if (p.gate && r < nq) {
      if (p.gate_wide) grow = p.gate + tok * p.ldg + head * p.V;
      else inv *= mtc_sigmoid(__bfloat162float(p.gate[tok * p.ldg + head]));
    }
    __nv_bfloat16* orow = p.y + tok * p.ldy + head * p.V;
#pragma unroll
    for (int c = 0; c < VP / 64; ++c) {
      uint32_t t[32];
      tmem_ld_32x32b_x32(o_addr + c * 32, t);
      tmem_ld_wait();
      const int col = half * (VP / 2) + c * 32;
      if (r < nq) {
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          if (col + i < p.V) {
            float f[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(t[i + e]) * inv;
            if (grow) {
              const uint4 raw = *reinterpret_cast<const uint4*>(grow + col + i);
              const uint32_t w4[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const float2 gg = unpack_bf16(w4[e]);
                f[2 * e] *= mtc_sigmoid(gg.x); f[2 * e + 1] *= mtc_sigmoid(gg.y);
              }
            }
            *reinterpret_cast<uint4*>(orow + col + i) = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
          }
        }
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (*stop) {                                                          // copies in flight land before the shared memory goes away
    for (int i = 0; i < 1000; ++i) __nanosleep(1000);
    if (threadIdx.x == 0) { *const_cast<volatile int*>(p.err) = 1; __threadfence_system(); }
    __syncthreads();
  }
  if (warp_idx == 1) {
    tc_fence_after_sync();
    tmem_dealloc<Cfg::TMEM_COLS>(tmem_base);
  }
}

template <int DC, int VP>
static cudaError_t launch_masked_attention_tc(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const MtcParams& p, int ntiles,
                                              cudaStream_t s) {
  auto kern = masked_attention_tc_kernel<DC, VP>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, MtcCfg<DC, VP>::SMEM_BYTES);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  kern<<<dim3((unsigned)p.H, (unsigned)ntiles), MTC_THREADS, MtcCfg<DC, VP>::SMEM_BYTES, s>>>(tq, tk, tv, p);
  return cudaGetLastError();
}

}  // namespace lb

// q [tokens, H*D]; kmat / vmat [rows, G*D] / [rows, G*V] with one row stride; the row of position p >= cstart[b] of sequence b is
// ext_off[b] + nsink[b] + p - cstart[b]; query tiles of 128.  Returns 0, a CUDA error code, or a negative code for sizes the kernel is not built for
extern "C" int lb_masked_attention_tc(const void* q, long ldq, const void* kmat, const void* vmat, long ldkv, const int* ext_off, const int* nsink, const int* cstart,
                                      const void* gate, long ldg, int gate_wide, const int* qt_seq, const int* qt_start, int ntiles,
                                      const int* seq_off, const int* past, void* y, long ldy, long tokens, long rows, int H, int G, int D, int V,
                                      int window, int chunk, float scale, float out_scale, float temp_coef, float temp_every, int* err, cudaStream_t s) {
  if (ntiles == 0) return 0;
  if (D < 16 || D > 128 || D % 16 || V < 16 || V > 128 || V % 16 || G < 1 || H % G || ntiles > 65535 || !(scale > 0.f) || temp_coef < 0.f) return -1;
  auto bad = [](const void* p, long ld) { return (reinterpret_cast<uintptr_t>(p) & 15) != 0 || ld % 8 != 0; };
  if (bad(q, ldq) || bad(kmat, ldkv) || bad(vmat, ldkv) || bad(y, ldy) || (gate && gate_wide && bad(gate, ldg))) return -3;
  CUtensorMap tq, tk, tv;
  {
    uint64_t dims[3] = {(uint64_t)D, (uint64_t)H, (uint64_t)tokens};
    uint64_t strides[3] = {2, (uint64_t)D * 2, (uint64_t)ldq * 2};
    uint32_t box[3] = {64, 1, 128};
    if (!lb_host::make_tmap_bf16(&tq, q, 3, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -2;
  }
  auto rows2d = [&](CUtensorMap* m, const void* base, long cols) {
    uint64_t dims[2] = {(uint64_t)cols, (uint64_t)rows};
    uint64_t strides[2] = {2, (uint64_t)ldkv * 2};
    uint32_t box[2] = {64, 128};
    return lb_host::make_tmap_bf16(m, base, 2, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B);
  };
  if (!rows2d(&tk, kmat, (long)G * D) || !rows2d(&tv, vmat, (long)G * V)) return -2;
  lb::MtcParams p{reinterpret_cast<__nv_bfloat16*>(y), ldy, reinterpret_cast<const __nv_bfloat16*>(gate), ldg, qt_seq, qt_start, seq_off, past, ext_off,
                  nsink, cstart, H, G, D, V, window, chunk, gate_wide, scale * 1.4426950408889634f, out_scale, temp_coef, temp_every, err};
  cudaError_t e;
  if (D <= 64) e = V <= 64 ? lb::launch_masked_attention_tc<1, 64>(tq, tk, tv, p, ntiles, s) : lb::launch_masked_attention_tc<1, 128>(tq, tk, tv, p, ntiles, s);
  else e = V <= 64 ? lb::launch_masked_attention_tc<2, 64>(tq, tk, tv, p, ntiles, s) : lb::launch_masked_attention_tc<2, 128>(tq, tk, tv, p, ntiles, s);
  return e == cudaSuccess ? 0 : (int)e;
}
