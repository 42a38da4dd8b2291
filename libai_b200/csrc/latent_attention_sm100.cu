// Prompt attention on expanded latents for sm_100a on tcgen05 / TMEM / TMA (bf16): per head D unrotated and R rotated query / key
// channels (D = 64 or 128, R <= 64), the rotated key part shared by all heads, values of V = 64 or 128, causal over ragged
// sequences that may continue a cached past, an optional number per head in the softmax denominator.
//
// One CTA per (head, tile of 128 consecutive queries of one sequence), 320 threads:
//   warp 0        TMA producer : the query tile once ([D | R | zeros] in 64-channel chunks), then key tiles of 128 keys — D / 64
//                                chunks of the head's own keys and one chunk of the shared part, which comes from the latent rows —
//                                and value tiles, both double buffered
//   warp 1        MMA issuer   : S = Q K^T into TMEM, O += P V with P read from TMEM
//   warps 2..9    softmax      : first rotate the query tile's last chunk in (swizzled) shared memory — the interleaved pairs of a
//                                row lie in the same 16-byte units — then two threads per query row: online softmax, P (bf16) to
//                                TMEM, the output kept in TMEM and rescaled only when the running maximum grows by more than 2^8
// Every wait on an mbarrier is bounded: when one runs out, the CTA stops issuing copies and products, runs its (finite) loops to
// the end without waiting, lets the copies in flight land, frees its TMEM and reports through `err`.
#include "attention_tc.cuh"

#include <type_traits>

namespace lb {

constexpr int LTC_BM = 128, LTC_BN = 128, LTC_THREADS = 320;

template <int DC, int V>     // DC: 64-channel chunks of the unrotated part
struct LtcCfg {
  static constexpr int CHUNK = 128 * 128;                               // 128 rows x 64 bf16
  static constexpr int Q_BYTES = (DC + 1) * CHUNK, K_BYTES = Q_BYTES, V_BYTES = (V / 64) * CHUNK;
  static constexpr int XCHG_BYTES = 2 * 2 * 128 * 4;                    // row maxima exchanged between the two halves: [parity][half][row]
  static constexpr int SMEM_BYTES = Q_BYTES + 2 * K_BYTES + 2 * V_BYTES + XCHG_BYTES + 1024 + 256;
  static constexpr uint32_t TMEM_COLS = V == 64 ? 256 : 512;
  static constexpr uint32_t S_COL = 0, O_COL = 128, P_COL = 128 + V;
};

struct LtcParams {
  __nv_bfloat16* y;
  long ldy;
  const float2* cs;          // [rows, R / 2] cos, sin
  const float* sink;         // [H] or null
  const int *qt_seq, *qt_start, *seq_off, *past, *ext_off;
  int D, R;
  float scale_log2;
  int* err;                  // mapped host word, set when a wait ran out
};

template <int DC, int V>
__global__ void __launch_bounds__(LTC_THREADS, 1)
latent_prompt_tc_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                        const __grid_constant__ CUtensorMap tmap_r, const __grid_constant__ CUtensorMap tmap_v, LtcParams p) {
  using Cfg = LtcCfg<DC, V>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + Cfg::Q_BYTES;
  uint8_t* sV = sK + 2 * Cfg::K_BYTES;
  float* sXchg = reinterpret_cast<float*>(sV + 2 * Cfg::V_BYTES);
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + 2 * Cfg::V_BYTES + Cfg::XCHG_BYTES);
  uint64_t *q_full = bars, *q_ready = bars + 1, *k_full = bars + 2, *k_empty = bars + 4, *v_full = bars + 6, *v_empty = bars + 8;
  uint64_t *s_full = bars + 10, *p_full = bars + 11, *o_full = bars + 12, *s_free = bars + 13;
  uint32_t* tmem_ptr_smem = reinterpret_cast<uint32_t*>(bars + 14);
  volatile int* stop = reinterpret_cast<volatile int*>(bars + 15);

  const int warp_idx = threadIdx.x / 32, lane = threadIdx.x % 32;
  const int head = blockIdx.x, b = p.qt_seq[blockIdx.y], t0 = p.qt_start[blockIdx.y];
  const int tok0 = p.seq_off[b] + t0, nq = min(LTC_BM, p.seq_off[b + 1] - tok0);
  const int pos0 = p.past[b] + t0, e0 = p.ext_off[b];
  const int nkv = (pos0 + nq + LTC_BN - 1) / LTC_BN;                    // key tiles up to the tile's last query

  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmap_q);
    tma_prefetch_desc(&tmap_k);
    tma_prefetch_desc(&tmap_r);
    tma_prefetch_desc(&tmap_v);
    mbar_init(q_full, 1);
    mbar_init(q_ready, 8);
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
      for (int c = 0; c <= DC; ++c) tma_load_3d(sQ + c * Cfg::CHUNK, &tmap_q, q_full, c * 64, head, tok0);
      for (int j = 0; j < nkv; ++j) {
        const int s = j & 1, row = e0 + j * LTC_BN;
        const uint32_t par = ((j >> 1) & 1) ^ 1;
        if (tc_wait(&k_empty[s], par, stop)) {
          mbar_arrive_expect_tx(&k_full[s], Cfg::K_BYTES);
#pragma unroll
          for (int c = 0; c < DC; ++c) tma_load_2d(sK + s * Cfg::K_BYTES + c * Cfg::CHUNK, &tmap_k, &k_full[s], head * (DC * 64) + c * 64, row);
          tma_load_2d(sK + s * Cfg::K_BYTES + DC * Cfg::CHUNK, &tmap_r, &k_full[s], 0, row);
        }
        if (tc_wait(&v_empty[s], par, stop)) {
          mbar_arrive_expect_tx(&v_full[s], Cfg::V_BYTES);
#pragma unroll
          for (int c = 0; c < V / 64; ++c) tma_load_2d(sV + s * Cfg::V_BYTES + c * Cfg::CHUNK, &tmap_v, &v_full[s], head * V + c * 64, row);
        }
      }
    }
    __syncwarp();
  } else if (warp_idx == 1) {
    constexpr uint32_t idesc_qk = make_idesc_bf16(LTC_BM, LTC_BN, false, false);
    constexpr uint32_t idesc_pv = make_idesc_bf16(LTC_BM, V, false, true);
    const uint32_t q_addr = smem_u32(sQ);
    const int rsteps = (p.R + 15) / 16;
    bool ok = __all_sync(0xffffffffu, tc_wait(q_ready, 0, stop));
    // S(j + 1) is issued as soon as the softmax warps have read S(j) for the last time, ahead of P(j) V(j)
    auto issue_qk = [&](int j) {
      const int s = j & 1;
      ok = __all_sync(0xffffffffu, ok && tc_wait(&k_full[s], (j >> 1) & 1, stop));
      if (j > 0) ok = __all_sync(0xffffffffu, ok && tc_wait(s_free, (j - 1) & 1, stop));
      tc_fence_after_sync();
      if (ok && elect_one()) {
        const uint32_t k_addr = smem_u32(sK + s * Cfg::K_BYTES);
#pragma unroll
        for (int kk = 0; kk < (DC + 1) * 4; ++kk) {
          if (kk < DC * 4 + rsteps) {
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
        for (int kk = 0; kk < LTC_BN / 16; ++kk)
          umma_f16_ts(tmem_base + Cfg::O_COL, tmem_base + Cfg::P_COL + kk * 8,
                      make_smem_desc_sw128(v_addr + kk * (16 * 128), LTC_BN * 128, 1024), idesc_pv, (j > 0 || kk > 0) ? 1u : 0u);
        umma_commit(o_full);
        umma_commit(&v_empty[s]);
      }
      __syncwarp();
    }
  } else {
    const int quad = warp_idx % 4, half = (warp_idx - 2) / 4;           // this warp's 64 of the 128 key columns
    const int r = quad * 32 + lane;                                     // query row of this thread (shared with the other half's thread)
    // ---- rotate the last query chunk in place: 16-byte unit u of row r sits at u ^ (r & 7)
    tc_wait(q_full, 0, stop);
    if (r < nq) {
      uint8_t* row = sQ + DC * Cfg::CHUNK + r * 128;
      const float2* cs = p.cs + static_cast<long>(tok0 + r) * (p.R / 2);
      for (int u = half; u < p.R / 8; u += 2) {
        uint4* at = reinterpret_cast<uint4*>(row + ((u ^ (r & 7)) << 4));
        uint4 w = *at;
        uint32_t* w4 = &w.x;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 t = cs[u * 4 + e], f = unpack_bf16(w4[e]);
          w4[e] = pack_bf16(f.x * t.x - f.y * t.y, f.y * t.x + f.x * t.y);
        }
        *at = w;
      }
    }
    fence_proxy_async();
    __syncwarp();
    if (lane == 0) mbar_arrive(q_ready);

    const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t s_addr = tmem_base + lane_off + Cfg::S_COL + half * 64;
    const uint32_t p_addr = tmem_base + lane_off + Cfg::P_COL + half * 32;
    const uint32_t o_addr = tmem_base + lane_off + Cfg::O_COL + half * (V / 2);
    float m_run = -INFINITY, l_run = 0.f;                               // log2 domain; l_run: the sum over this half's columns
    const int key_lim = pos0 + r + 1;                                   // keys [0, key_lim) are visible to this row
    for (int j = 0; j < nkv; ++j) {
      tc_wait(s_full, j & 1, stop);
      __syncwarp();
      tc_fence_after_sync();
      const int k0 = j * LTC_BN + half * 64;
      const bool need_mask = j * LTC_BN + LTC_BN > pos0 + 1;            // some row of the tile does not see the whole key tile
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
            if constexpr (MASK) x = k0 + c * 32 + i < key_lim ? x : -INFINITY;
            mx = fmaxf(mx, x);
          }
        }
      };
      if (need_mask) pass1(std::true_type{}); else pass1(std::false_type{});
      float* xch = sXchg + (j & 1) * 256;
      xch[half * 128 + r] = mx;
      tc_pair_sync(quad);
      mx = fmaxf(mx, xch[(half ^ 1) * 128 + r]);
      const float m_cand = fmaxf(m_run, mx * p.scale_log2);
      const bool bump = (m_cand - m_run > 8.0f) || (m_run == -INFINITY && m_cand != -INFINITY);
      float alpha = 1.0f;
      if (bump) { alpha = fast_exp2(m_run - m_cand); m_run = m_cand; }  // 0 on the first tile
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
            float x0 = fast_exp2(__uint_as_float(t[i]) * p.scale_log2 - m_use), x1 = fast_exp2(__uint_as_float(t[i + 1]) * p.scale_log2 - m_use);
            if constexpr (MASK) {
              const int kidx = k0 + c * 32 + i;
              x0 = kidx < key_lim ? x0 : 0.f;
              x1 = kidx + 1 < key_lim ? x1 : 0.f;
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
        for (int c = 0; c < V / 64; ++c) {
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
    if (p.sink) l_run += fast_exp2(p.sink[head] * 1.4426950408889634f - m_run);
    tc_wait(o_full, (nkv - 1) & 1, stop);
    __syncwarp();
    tc_fence_after_sync();
    const float inv = l_run > 0.f ? 1.0f / l_run : 0.f;
    __nv_bfloat16* orow = p.y + static_cast<long>(tok0 + r) * p.ldy + head * V + half * (V / 2);
#pragma unroll
    for (int c = 0; c < V / 64; ++c) {
      uint32_t t[32];
      tmem_ld_32x32b_x32(o_addr + c * 32, t);
      tmem_ld_wait();
      if (r < nq) {
#pragma unroll
        for (int i = 0; i < 32; i += 8)
          *reinterpret_cast<uint4*>(orow + c * 32 + i) = make_uint4(
              pack_bf16(__uint_as_float(t[i]) * inv, __uint_as_float(t[i + 1]) * inv), pack_bf16(__uint_as_float(t[i + 2]) * inv, __uint_as_float(t[i + 3]) * inv),
              pack_bf16(__uint_as_float(t[i + 4]) * inv, __uint_as_float(t[i + 5]) * inv), pack_bf16(__uint_as_float(t[i + 6]) * inv, __uint_as_float(t[i + 7]) * inv));
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

template <int DC, int V>
static cudaError_t launch_latent_prompt_tc(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tr, const CUtensorMap& tv, const LtcParams& p,
                                           int H, int ntiles, cudaStream_t s) {
  auto kern = latent_prompt_tc_kernel<DC, V>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, LtcCfg<DC, V>::SMEM_BYTES);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  kern<<<dim3((unsigned)H, (unsigned)ntiles), LTC_THREADS, LtcCfg<DC, V>::SMEM_BYTES, s>>>(tq, tk, tr, tv, p);
  return cudaGetLastError();
}

}  // namespace lb

// q [tokens, ldq] (per head [D | R], R unrotated), kv [rows, ldkv] = [H*D keys | H*V values], rot [rows, ldr] = the shared rotated key
// part (R numbers per row); returns 0, a CUDA error code, or a negative code for sizes the kernel is not built for
extern "C" int lb_latent_prompt_tc(const void* q, long ldq, const void* kv, long ldkv, const void* rot, long ldr, const float* cs, const float* sink,
                                   const int* ext_off, const int* qt_seq, const int* qt_start, int ntiles, const int* seq_off, const int* past, void* y,
                                   long ldy, long tokens, long rows, int H, int D, int R, int V, float scale, int* err, cudaStream_t s) {
  if (ntiles == 0) return 0;
  if ((D != 64 && D != 128) || (V != 64 && V != 128) || R < 8 || R > 64 || R % 8 || ntiles > 65535) return -1;
  auto bad = [](const void* p, long ld) { return (reinterpret_cast<uintptr_t>(p) & 15) != 0 || ld % 8 != 0; };
  if (bad(q, ldq) || bad(kv, ldkv) || bad(rot, ldr) || bad(y, ldy) || (reinterpret_cast<uintptr_t>(cs) & 7) != 0) return -3;
  const __nv_bfloat16* kvb = reinterpret_cast<const __nv_bfloat16*>(kv);
  CUtensorMap tq, tk, tr, tv;
  {
    uint64_t dims[3] = {(uint64_t)(D + R), (uint64_t)H, (uint64_t)tokens};
    uint64_t strides[3] = {2, (uint64_t)(D + R) * 2, (uint64_t)ldq * 2};
    uint32_t box[3] = {64, 1, 128};
    if (!lb_host::make_tmap_bf16(&tq, q, 3, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B)) return -2;
  }
  auto rows2d = [&](CUtensorMap* m, const void* base, long cols, long ld) {
    uint64_t dims[2] = {(uint64_t)cols, (uint64_t)rows};
    uint64_t strides[2] = {2, (uint64_t)ld * 2};
    uint32_t box[2] = {64, 128};
    return lb_host::make_tmap_bf16(m, base, 2, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B);
  };
  if (!rows2d(&tk, kvb, (long)H * D, ldkv) || !rows2d(&tr, rot, R, ldr) || !rows2d(&tv, kvb + (long)H * D, (long)H * V, ldkv)) return -2;
  lb::LtcParams p{reinterpret_cast<__nv_bfloat16*>(y), ldy, reinterpret_cast<const float2*>(cs), sink, qt_seq, qt_start, seq_off, past, ext_off, D, R,
                  scale * 1.4426950408889634f, err};
  cudaError_t e;
  if (D == 64) e = V == 64 ? lb::launch_latent_prompt_tc<1, 64>(tq, tk, tr, tv, p, H, ntiles, s) : lb::launch_latent_prompt_tc<1, 128>(tq, tk, tr, tv, p, H, ntiles, s);
  else e = V == 64 ? lb::launch_latent_prompt_tc<2, 64>(tq, tk, tr, tv, p, H, ntiles, s) : lb::launch_latent_prompt_tc<2, 128>(tq, tk, tr, tv, p, H, ntiles, s);
  return e == cudaSuccess ? 0 : (int)e;
}
