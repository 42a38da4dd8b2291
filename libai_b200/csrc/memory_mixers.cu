// Prompts through a matrix memory with exponential gates (memory_gates_kernel of lin_mixers.cu has the recurrence), chunk by chunk on the
// tensor cores (bf16 operands, fp32 accumulation).  With F_t the sum of the log forget gates f from the chunk's start, i the log input
// gates, m the running maximum and m_0 its value before the chunk:
//   c_ts = exp(F_t - F_s + i_s - m_t)  (s <= t),   A_t = exp(F_t + m_0 - m_t),
//   S^T q -> A_t S_0^T q_t + sum_s c_ts (q_t . k_s) v_s,     z . q -> A_t z_0 . q_t + sum_s c_ts (q_t . k_s),
//   S <- A_L S_0 + sum_s c_Ls k_s v_s^T,                     z <- A_L z_0 + sum_s c_Ls k_s,
// which is what the token-by-token recurrence gives.  fp32 factors never enter a product rounded: the state, the weighted scores and the
// weighted keys are each written as a sum of three bf16 numbers (24 bits), and the products of the parts are added up in fp32.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

namespace {

using bf16 = __nv_bfloat16;
constexpr int MC_L = 64;               // tokens per chunk
constexpr int MC_THREADS = 256;        // warp w: query rows / key channels of group w & 3, value columns of half w >> 2
constexpr int MC_GATES = 6;            // F (upper part), F (rest), i, m, A, exp(-m)

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x2_trans(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];\n" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float2 unpack2(uint32_t u) { return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u)); }
// a pair of fp32 numbers as three pairs of bf16 numbers that add up to them
__device__ __forceinline__ void split3(float x, float y, uint32_t (&p)[3]) {
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    p[i] = pack2(x, y);
    const float2 t = unpack2(p[i]);
    x -= t.x; y -= t.y;
  }
}
// the output gate's activation, rounded to bf16 with the result
__device__ __forceinline__ float sigmoid1(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

template <int DB, int NB>              // DB: key channels / 16 (padded), NB: blocks of 8 value columns per warp
struct McCfg {
  static constexpr int DP = DB * 16, VT = 2 * NB * 8, MB = DB >= 4 ? DB / 4 : 1;
  static constexpr int QS = DP + 8, VS = VT + 8;                         // row strides: an odd number of 16-byte units
  static constexpr int STAGE = 2 * MC_L * QS + MC_L * VS;                // bf16 numbers of one [Q | K | V] stage
  static constexpr int STATE = 3 * DP * VS;                              // the state's three parts; columns VT .. VT + 7 hold z
  static constexpr int SMEM = (2 * STAGE + STATE) * 2 + 2 * MC_GATES * MC_L * 4 + 2 * MC_L * 4;
};

template <int DB, int NB>
__global__ void __launch_bounds__(MC_THREADS, 1)
memory_chunk_kernel(const bf16* __restrict__ q, long ldq, const bf16* __restrict__ k, long ldk, const bf16* __restrict__ v, long ldv,
                    const float* __restrict__ gates, float q_scale, float* __restrict__ S, float* Z, float* ztmp,
                    const int* __restrict__ seq_off, const int* __restrict__ slots, const int* __restrict__ past, float* __restrict__ out,
                    const bf16* __restrict__ w, const bf16* __restrict__ gate, long ldg, float eps, float out_scale, bf16* __restrict__ y, long ldy,
                    long tokens, int H, int D, int V) {
  using Cfg = McCfg<DB, NB>;
  constexpr int DP = Cfg::DP, VT = Cfg::VT, MB = Cfg::MB, QS = Cfg::QS, VS = Cfg::VS;
  extern __shared__ __align__(16) unsigned char mc_smem[];
  bf16* const stages = reinterpret_cast<bf16*>(mc_smem);
  bf16* const sS = stages + 2 * Cfg::STAGE;
  float* const sG = reinterpret_cast<float*>(sS + Cfg::STATE);          // [2][MC_GATES][64]
  float* const sR = sG + 2 * MC_GATES * MC_L;                           // [2 column halves][64]: sums of squares of the rows
  const int b = blockIdx.x / H, h = blockIdx.x - b * H, j0 = blockIdx.y * VT;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;
  const int wr = warp & 3, wc = warp >> 2, cw = wc * NB * 8;            // this warp's first value column within the block's
  const long tok0 = seq_off[b];
  const int n = seq_off[b + 1] - seq_off[b];
  const bool cont = past[b] > 0, owner = DB >= 4 || wr < DB;            // owner: this warp holds rows of the state
  float* const Sg = S + ((long)slots[b] * H + h) * (long)D * V;
  float* const Zg = Z + ((long)slots[b] * H + h) * D;
  const float* const gh = gates + (long)h * MC_GATES * tokens;

  // ---- the state: fp32 accumulator fragments, rows (wr * MB + i) * 16 + gid (+ 8), columns j0 + cw + 8 nb + 2 tig (+ 1)
  float s[MB][NB][4], z[MB][2];
#pragma unroll
  for (int i = 0; i < MB; ++i) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int d = (wr * MB + i) * 16 + gid + 8 * e;
      const bool row = cont && owner && d < D;
      z[i][e] = row ? Zg[d] : 0.f;
#pragma unroll
      for (int nb = 0; nb < NB; ++nb) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const int col = j0 + cw + nb * 8 + tig * 2 + c;
          s[i][nb][2 * e + c] = (row && col < V) ? Sg[(long)d * V + col] : 0.f;
        }
      }
    }
  }
  auto store_parts = [&]() {                                            // the state's three bf16 parts to shared memory
    if (owner) {
#pragma unroll
      for (int i = 0; i < MB; ++i) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int d = (wr * MB + i) * 16 + gid + 8 * e;
          uint32_t p[3];
#pragma unroll
          for (int nb = 0; nb < NB; ++nb) {
            split3(s[i][nb][2 * e], s[i][nb][2 * e + 1], p);
#pragma unroll
            for (int t = 0; t < 3; ++t) *reinterpret_cast<uint32_t*>(sS + ((long)t * DP + d) * VS + cw + nb * 8 + tig * 2) = p[t];
          }
          if (wc == 0) {                                                // z in the first of the eight columns after the values, zeros beside it
            split3(tig == 0 ? z[i][e] : 0.f, 0.f, p);
#pragma unroll
            for (int t = 0; t < 3; ++t) *reinterpret_cast<uint32_t*>(sS + ((long)t * DP + d) * VS + VT + tig * 2) = p[t];
          }
        }
      }
    }
  };
  auto prefetch = [&](int c0) {                                         // tokens c0 .. c0 + 63 of the step to the stage of their chunk
    const int st = (c0 / MC_L) & 1;
    bf16* const dq = stages + st * Cfg::STAGE;
    bf16* const dk = dq + MC_L * QS;
    bf16* const dv = dk + MC_L * QS;
    for (int i = tid; i < MC_L * (DP / 8); i += MC_THREADS) {
      const int r = i / (DP / 8), ch = (i - r * (DP / 8)) * 8;
      const bool ok = c0 + r < n && ch < D;
      const long row = tok0 + (ok ? c0 + r : 0);
      const int col = h * D + (ok ? ch : 0);
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_u32(dq + r * QS + ch)), "l"(q + row * ldq + col), "r"(ok ? 16 : 0));
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_u32(dk + r * QS + ch)), "l"(k + row * ldk + col), "r"(ok ? 16 : 0));
    }
    for (int i = tid; i < MC_L * (VT / 8); i += MC_THREADS) {
      const int r = i / (VT / 8), ch = (i - r * (VT / 8)) * 8;
      const bool ok = c0 + r < n && j0 + ch < V;
      const bf16* src = v + (tok0 + (ok ? c0 + r : 0)) * ldv + h * V + (ok ? j0 + ch : 0);
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(smem_u32(dv + r * VS + ch)), "l"(src), "r"(ok ? 16 : 0));
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
    // gates: tokens beyond the step write nothing (i = -inf) and leave F and m where they are
    for (int i = tid; i < MC_GATES * MC_L; i += MC_THREADS) {
      const int a = i / MC_L, t = i - a * MC_L, last = min(t, n - 1 - c0);
      sG[st * MC_GATES * MC_L + i] = (a == 2 && last < t) ? -INFINITY : gh[(long)a * tokens + tok0 + c0 + last];
    }
  };
  store_parts();
  prefetch(0);
  uint32_t wv[NB];                                                      // weights of this thread's columns (fused read-out)
#pragma unroll
  for (int nb = 0; nb < NB; ++nb) {
    const int col = cw + nb * 8 + tig * 2;
    wv[nb] = (y && w && col < V) ? *reinterpret_cast<const uint32_t*>(w + h * V + col) : 0x3f803f80u;
  }
  const int r0 = wr * 16 + gid, r1 = r0 + 8;                            // this thread's two query rows within the chunk
  for (int c0 = 0; c0 < n; c0 += MC_L) {
    const int st = (c0 / MC_L) & 1;
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();                                                    // the chunk, its gates and the state's parts are in place; nobody reads the other stage
    if (c0 + MC_L < n) prefetch(c0 + MC_L);
    const bf16* const sQ = stages + st * Cfg::STAGE;
    const bf16* const sK = sQ + MC_L * QS;
    const bf16* const sV = sK + MC_L * QS;
    const float* const g = sG + st * MC_GATES * MC_L;
    const bool ok0 = c0 + r0 < n, ok1 = c0 + r1 < n;
    uint32_t gv0[NB], gv1[NB];                                          // output gates of the two rows
    if (y) {
#pragma unroll
      for (int nb = 0; nb < NB; ++nb) {
        const int col = cw + nb * 8 + tig * 2;
        const bf16* gp = gate + (tok0 + c0) * ldg + h * V + col;
        gv0[nb] = (gate && ok0 && col < V) ? *reinterpret_cast<const uint32_t*>(gp + r0 * ldg) : 0u;
        gv1[nb] = (gate && ok1 && col < V) ? *reinterpret_cast<const uint32_t*>(gp + r1 * ldg) : 0u;
      }
    }
    float o[NB][4], zq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) { o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.f; }
    float sc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) { sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f; }
    // ---- q S_0 (and q . z_0), q k
    const uint32_t qrow = smem_u32(sQ + (wr * 16 + (lane & 15)) * QS + (lane >> 4) * 8);
    const uint32_t krow = smem_u32(sK + ((lane >> 4) * 8 + (lane & 7)) * QS + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int kk = 0; kk < DB; ++kk) {
      uint32_t qf[4];
      ldsm_x4(qf, qrow + kk * 32);
#pragma unroll
      for (int t = 0; t < 3; ++t) {
        const uint32_t srow = smem_u32(sS + (t * DP + kk * 16 + (lane & 15)) * VS + (lane >> 4) * 8);
#pragma unroll
        for (int nb = 0; nb < NB; nb += 2) {
          uint32_t bb[4];
          ldsm_x4_trans(bb, srow + (cw + nb * 8) * 2);
          mma_bf16(o[nb], qf, bb[0], bb[1]);
          mma_bf16(o[nb + 1], qf, bb[2], bb[3]);
        }
        uint32_t b0, b1;
        ldsm_x2_trans(b0, b1, smem_u32(sS + (t * DP + kk * 16 + (lane & 15)) * VS + VT));
        mma_bf16(zq, qf, b0, b1);
      }
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        if (j < 2 * wr + 2) {                                           // keys up to the warp's last row
          uint32_t bb[4];
          ldsm_x4(bb, krow + (j * 8 * QS + kk * 16) * 2);
          mma_bf16(sc[j], qf, bb[0], bb[1]);
          mma_bf16(sc[j + 1], qf, bb[2], bb[3]);
        }
      }
    }
    const float A0 = g[4 * MC_L + r0], A1 = g[4 * MC_L + r1];
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) { o[nb][0] *= A0; o[nb][1] *= A0; o[nb][2] *= A1; o[nb][3] *= A1; }
    // ---- weights c_ts and their row sums
    const float fh0 = g[r0], fl0 = g[MC_L + r0], m0 = g[3 * MC_L + r0], fh1 = g[r1], fl1 = g[MC_L + r1], m1 = g[3 * MC_L + r1];
    float p0 = 0.f, p1 = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (j < 2 * wr + 2) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const int t = j * 8 + tig * 2 + c;
          const float fh = g[t], fl = g[MC_L + t], li = g[2 * MC_L + t];
          sc[j][c] = t <= r0 ? sc[j][c] * expf(((fh0 - fh) + (fl0 - fl)) + (li - m0)) : 0.f;
          sc[j][2 + c] = t <= r1 ? sc[j][2 + c] * expf(((fh1 - fh) + (fl1 - fl)) + (li - m1)) : 0.f;
          p0 += sc[j][c]; p1 += sc[j][2 + c];
        }
      }
    }
    p0 += __shfl_xor_sync(0xffffffffu, p0, 1); p0 += __shfl_xor_sync(0xffffffffu, p0, 2);
    p1 += __shfl_xor_sync(0xffffffffu, p1, 1); p1 += __shfl_xor_sync(0xffffffffu, p1, 2);
    const float z0 = __shfl_sync(0xffffffffu, zq[0], lane & 28), z1 = __shfl_sync(0xffffffffu, zq[2], lane & 28);
    const float d0 = q_scale / (fmaxf(fabsf((A0 * z0 + p0) * q_scale), g[5 * MC_L + r0]) + 1e-6f);
    const float d1 = q_scale / (fmaxf(fabsf((A1 * z1 + p1) * q_scale), g[5 * MC_L + r1]) + 1e-6f);
    // ---- o += c v,  S <- A_L S + (c_L k)^T v  on the same value fragments
    const float AL = g[4 * MC_L + 63], fhL = g[63], flL = g[MC_L + 63], mL = g[3 * MC_L + 63];
#pragma unroll
    for (int i = 0; i < MB; ++i) {
#pragma unroll
      for (int nb = 0; nb < NB; ++nb) { s[i][nb][0] *= AL; s[i][nb][1] *= AL; s[i][nb][2] *= AL; s[i][nb][3] *= AL; }
    }
    float zs[MB][2];
#pragma unroll
    for (int i = 0; i < MB; ++i) zs[i][0] = zs[i][1] = 0.f;
#pragma unroll
    for (int k2 = 0; k2 < 4; ++k2) {
      const int t = k2 * 16 + tig * 2;
      float cl[4];                                                      // c_Ls of the tokens t, t + 1, t + 8, t + 9
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int u = t + (e >> 1) * 8 + (e & 1);
        cl[e] = expf(((fhL - g[u]) + (flL - g[MC_L + u])) + (g[2 * MC_L + u] - mL));
      }
      uint32_t ka[MB][3][4];
      if (owner) {
#pragma unroll
        for (int i = 0; i < MB; ++i) {
          uint32_t kf[4];
          ldsm_x4_trans(kf, smem_u32(sK + (k2 * 16 + (lane >> 4) * 8 + (lane & 7)) * QS + (wr * MB + i) * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
          for (int e = 0; e < 4; ++e) {                                 // e: rows gid / gid + 8 (bit 0), tokens t / t + 8 (bit 1)
            const float2 x = unpack2(kf[e]);
            const float a = x.x * cl[(e >> 1) * 2], c = x.y * cl[(e >> 1) * 2 + 1];
            zs[i][e & 1] += a + c;
            uint32_t parts[3];
            split3(a, c, parts);
#pragma unroll
            for (int u = 0; u < 3; ++u) ka[i][u][e] = parts[u];
          }
        }
      }
      uint32_t pa[3][4];
      if (k2 <= wr) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          uint32_t parts[3];
          split3(sc[2 * k2 + (e >> 1)][2 * (e & 1)], sc[2 * k2 + (e >> 1)][2 * (e & 1) + 1], parts);
#pragma unroll
          for (int u = 0; u < 3; ++u) pa[u][e] = parts[u];
        }
      }
      const uint32_t vrow = smem_u32(sV + (k2 * 16 + (lane & 15)) * VS + cw + (lane >> 4) * 8);
#pragma unroll
      for (int nb = 0; nb < NB; nb += 4) {                              // products of one part go to four accumulators in turn
        uint32_t ba[4], bb[4];
        ldsm_x4_trans(ba, vrow + nb * 16);
        ldsm_x4_trans(bb, vrow + nb * 16 + 32);
#pragma unroll
        for (int u = 0; u < 3; ++u) {
          if (k2 <= wr) {
            mma_bf16(o[nb], pa[u], ba[0], ba[1]); mma_bf16(o[nb + 1], pa[u], ba[2], ba[3]);
            mma_bf16(o[nb + 2], pa[u], bb[0], bb[1]); mma_bf16(o[nb + 3], pa[u], bb[2], bb[3]);
          }
          if (owner) {
#pragma unroll
            for (int i = 0; i < MB; ++i) {
              mma_bf16(s[i][nb], ka[i][u], ba[0], ba[1]); mma_bf16(s[i][nb + 1], ka[i][u], ba[2], ba[3]);
              mma_bf16(s[i][nb + 2], ka[i][u], bb[0], bb[1]); mma_bf16(s[i][nb + 3], ka[i][u], bb[2], bb[3]);
            }
          }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < MB; ++i) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float t = zs[i][e];
        t += __shfl_xor_sync(0xffffffffu, t, 1); t += __shfl_xor_sync(0xffffffffu, t, 2);
        z[i][e] = z[i][e] * AL + t;
      }
    }
    // ---- read-out
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) { o[nb][0] *= d0; o[nb][1] *= d0; o[nb][2] *= d1; o[nb][3] *= d1; }
    if (y) {
      float q0 = 0.f, q1 = 0.f;
#pragma unroll
      for (int nb = 0; nb < NB; ++nb) { q0 += o[nb][0] * o[nb][0] + o[nb][1] * o[nb][1]; q1 += o[nb][2] * o[nb][2] + o[nb][3] * o[nb][3]; }
      q0 += __shfl_xor_sync(0xffffffffu, q0, 1); q0 += __shfl_xor_sync(0xffffffffu, q0, 2);
      q1 += __shfl_xor_sync(0xffffffffu, q1, 1); q1 += __shfl_xor_sync(0xffffffffu, q1, 2);
      if (tig == 0) { sR[wc * MC_L + r0] = q0; sR[wc * MC_L + r1] = q1; }
    }
    __syncthreads();                                                    // everyone has read the state's parts; the rows' sums are complete
    store_parts();
    if (y) {
      const float i0 = out_scale / sqrtf((sR[r0] + sR[MC_L + r0]) / (float)V + eps), i1 = out_scale / sqrtf((sR[r1] + sR[MC_L + r1]) / (float)V + eps);
      bf16* yp = y + (tok0 + c0) * ldy + h * V;
#pragma unroll
      for (int nb = 0; nb < NB; ++nb) {
        const int col = cw + nb * 8 + tig * 2;
        if (col < V) {
          const float2 ww = unpack2(wv[nb]), g0 = unpack2(gv0[nb]), g1 = unpack2(gv1[nb]);
          const float a = gate ? sigmoid1(g0.x) : 1.f, c = gate ? sigmoid1(g0.y) : 1.f, e = gate ? sigmoid1(g1.x) : 1.f, f = gate ? sigmoid1(g1.y) : 1.f;
          if (ok0) *reinterpret_cast<uint32_t*>(yp + r0 * ldy + col) = pack2(o[nb][0] * i0 * ww.x * a, o[nb][1] * i0 * ww.y * c);
          if (ok1) *reinterpret_cast<uint32_t*>(yp + r1 * ldy + col) = pack2(o[nb][2] * i1 * ww.x * e, o[nb][3] * i1 * ww.y * f);
        }
      }
    } else {
      float* op = out + (tok0 + c0) * (long)(H * V) + h * V;
#pragma unroll
      for (int nb = 0; nb < NB; ++nb) {
        const int col = j0 + cw + nb * 8 + tig * 2;
        if (col < V) {
          if (ok0) *reinterpret_cast<float2*>(op + (long)r0 * H * V + col) = make_float2(o[nb][0], o[nb][1]);
          if (ok1) *reinterpret_cast<float2*>(op + (long)r1 * H * V + col) = make_float2(o[nb][2], o[nb][3]);
        }
      }
    }
  }
  if (owner) {
#pragma unroll
    for (int i = 0; i < MB; ++i) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = (wr * MB + i) * 16 + gid + 8 * e;
        if (d >= D) continue;
        // with several column blocks a block may start after this one ended, and must still read the old z
        if (wc == 0 && tig == 0 && blockIdx.y == 0) (gridDim.y > 1 ? ztmp + (long)blockIdx.x * D : Zg)[d] = z[i][e];
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) {
          const int col = j0 + cw + nb * 8 + tig * 2;
          if (col < V) *reinterpret_cast<float2*>(Sg + (long)d * V + col) = make_float2(s[i][nb][2 * e], s[i][nb][2 * e + 1]);
        }
      }
    }
  }
}

__global__ void memory_keysum_store_kernel(const float* __restrict__ ztmp, float* __restrict__ Z, const int* __restrict__ slots, int H, int D) {
  const int b = blockIdx.x / H, h = blockIdx.x - b * H;
  for (int i = threadIdx.x; i < D; i += blockDim.x) Z[((long)slots[b] * H + h) * D + i] = ztmp[(long)blockIdx.x * D + i];
}

template <int DB, int NB>
cudaError_t launch_chunks(dim3 grid, cudaStream_t st, const bf16* q, long ldq, const bf16* k, long ldk, const bf16* v, long ldv, const float* gates,
                          float q_scale, float* S, float* Z, float* ztmp, const int* seq_off, const int* slots, const int* past, float* out,
                          const bf16* w, const bf16* gate, long ldg, float eps, float out_scale, bf16* y, long ldy, long tokens, int H, int D, int V) {
  auto kern = memory_chunk_kernel<DB, NB>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, McCfg<DB, NB>::SMEM);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  kern<<<grid, MC_THREADS, McCfg<DB, NB>::SMEM, st>>>(q, ldq, k, ldk, v, ldv, gates, q_scale, S, Z, ztmp, seq_off, slots, past, out, w, gate, ldg,
                                                      eps, out_scale, y, ldy, tokens, H, D, V);
  return cudaGetLastError();
}

}  // namespace

extern "C" {

// whether the chunk kernel takes these operands; the number of blocks of value columns per head it would use (0: it does not)
int lbm_memory_chunk_blocks(const void* q, long ldq, const void* k, long ldk, const void* v, long ldv, int B, int H, int D, int V) {
  auto bad = [](const void* p, long ld) { return ((uintptr_t)p & 15) != 0 || ld % 8 != 0; };
  if (D % 8 || V % 8 || D < 8 || D > 128 || V < 8 || bad(q, ldq) || bad(k, ldk) || bad(v, ldv)) return 0;
  if (V <= 64) return 1;
  const int wide = (V + 127) / 128;
  return (long)B * H * wide < 75 ? (V + 63) / 64 : wide;               // few (sequence, head) pairs: narrower blocks for the idle SMs
}

// `blocks` as lbm_memory_chunk_blocks gave it; y given (one block of columns only): the normed, weighted, gated read-out in bf16, else
// out fp32 [tokens, H*V].  S must be 8-byte aligned with V even
int lbm_memory_chunk(const void* q, long ldq, const void* k, long ldk, const void* v, long ldv, const float* gates, float q_scale, float* S,
                     float* Z, float* ztmp, const int* seq_off, const int* slots, const int* past, float* out, const void* w, const void* gate,
                     long ldg, float eps, float out_scale, void* y, long ldy, long tokens, int B, int H, int D, int V, int blocks, cudaStream_t s) {
  if (B == 0 || tokens == 0) return 0;
  if (blocks < 1 || (y && blocks != 1) || (!y && !out) || D > 128) return -1;
  if (y && (ldy % 2 || ((uintptr_t)y & 3) || ((uintptr_t)w & 3) || (gate && (ldg % 2 || ((uintptr_t)gate & 3))))) return -1;
  const int per = (V + blocks - 1) / blocks;
  if (per > 128) return -1;
  const dim3 grid((unsigned)(B * H), (unsigned)blocks);
  cudaError_t e;
#define MCL(DBV, NBV) e = launch_chunks<DBV, NBV>(grid, s, (const bf16*)q, ldq, (const bf16*)k, ldk, (const bf16*)v, ldv, gates, q_scale, S, Z, ztmp, \
    seq_off, slots, past, out, (const bf16*)w, (const bf16*)gate, ldg, eps, out_scale, (bf16*)y, ldy, tokens, H, D, V)
  if (D <= 32) { if (per <= 64) MCL(2, 4); else MCL(2, 8); }
  else if (D <= 64) { if (per <= 64) MCL(4, 4); else MCL(4, 8); }
  else { if (per <= 64) MCL(8, 4); else MCL(8, 8); }
#undef MCL
  if (e == cudaSuccess && blocks > 1) {
    memory_keysum_store_kernel<<<(unsigned)(B * H), 128, 0, s>>>(ztmp, Z, slots, H, D);
    e = cudaGetLastError();
  }
  return e == cudaSuccess ? 0 : (int)e;
}

}  // extern "C"
