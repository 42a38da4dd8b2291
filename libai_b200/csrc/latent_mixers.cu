// Kernels of attention on paged low-rank latents with a shared rotated key part (multi-head latent attention over the whole past):
//   * preparation: RMS norm of the query latent; RMS norm of the key/value latent and rotation of the shared key part, both
//     written into the token's cache row; the step's cos / sin table;
//   * gather of a sequence's cache rows (a prompt portion that continues a sequence expands keys and values of all of them);
//   * prompt attention on expanded keys and values: a generic kernel and a tensor-core kernel (bf16);
//   * absorbed attention for single-token steps and short portions: the query is pulled through the key up-projection, scores and
//     the weighted sum run on the cached rows themselves (a generic kernel and a tensor-core kernel), and a last kernel merges the
//     parts of a sequence's keys and applies the value up-projection.
//
// Conventions (the ragged-batch descriptor of the other mixer libraries).  A step carries B sequences; row t of a step belongs to
// sequence b = tok_seq[t], its position is past[b] + t - seq_off[b], its state lives in slot slots[b].  A cache row is
// [C latent | R rotated key part | zero padding] (CS numbers, CS >= C + R); position p of a sequence lives in row p % page_size of
// page table[slot * max_pages + p / page_size] of the pool [pages, page_size, CS].  A head's query is [D unrotated | R rotated];
// rotation turns the channel pair (2i, 2i + 1) of the rotated part by position * freq[i] (i < half; later pairs pass unchanged) and
// multiplies it by a constant.  Queries arrive unrotated: the attention kernels rotate them while they load them, with the table
// cs [rows, R / 2] of (cos, sin).  Activations are `T` (float or bf16); angles, norms, scores and the softmax are fp32 in both.
// Built WITHOUT fast-math.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

namespace {
typedef __nv_bfloat16 bf16;

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<bf16>(const bf16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void stf(T* p, float v);
template <> __device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stf<bf16>(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int m = 16; m > 0; m >>= 1) v += __shfl_xor_sync(0xffffffffu, v, m);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int m = 16; m > 0; m >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, m));
  return v;
}

// VEC consecutive channels of a row (8 bf16 or 4 floats per 16-byte access; VEC = 1: anything)
template <typename T, int VEC> struct Pack;
template <typename T> struct Pack<T, 1> {
  static __device__ __forceinline__ void ld(const T* p, float (&f)[1]) { f[0] = ldf(p); }
  static __device__ __forceinline__ void st(T* p, const float (&f)[1]) { stf(p, f[0]); }
};
template <> struct Pack<float, 4> {
  static __device__ __forceinline__ void ld(const float* p, float (&f)[4]) { const float4 a = *reinterpret_cast<const float4*>(p); f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; }
  static __device__ __forceinline__ void st(float* p, const float (&f)[4]) { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};
template <> struct Pack<bf16, 8> {
  static __device__ __forceinline__ void ld(const bf16* p, float (&f)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) { const float2 t = __bfloat1622float2(h2[e]); f[2 * e] = t.x; f[2 * e + 1] = t.y; }
  }
  static __device__ __forceinline__ void st(bf16* p, const float (&f)[8]) {
    uint4 raw;
    __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) h2[e] = __floats2bfloat162_rn(f[2 * e], f[2 * e + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
  }
};

// ------------------------------------------------------------------------------------------------------------------
// Preparation.  One warp per (token, unit): unit 0 — the key/value latent and the shared key part (dkv row [C | R]) -> the
// token's page row, optionally a packed copy `lat` [rows, CS], and the token's cos / sin entries; unit 1 (when dq is given) —
// the query latent -> cq.  Norm: v / sqrt(mean(v^2) + eps) * w.
// ------------------------------------------------------------------------------------------------------------------
template <typename T, int VEC>
__device__ __forceinline__ float row_rms(const T* src, int n, float eps, int lane) {
  float ss = 0.f;
  for (int i = lane * VEC; i < n; i += 32 * VEC) {
    float f[VEC];
    Pack<T, VEC>::ld(src + i, f);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss += f[e] * f[e];
  }
  return 1.f / sqrtf(warp_sum(ss) / (float)n + eps);
}

template <typename T, int VEC>
__global__ void __launch_bounds__(128)
latent_prepare_kernel(const T* __restrict__ dkv, long ldk, const T* __restrict__ dq, long lddq, const T* __restrict__ wkv,
                      const T* __restrict__ wq, const float* __restrict__ freq, int half, float mscale, float eps, T* __restrict__ pool,
                      const int* __restrict__ table, int max_pages, int page_size, T* __restrict__ lat, T* __restrict__ cq,
                      float2* __restrict__ cs, const int* __restrict__ tok_seq, const int* __restrict__ seq_off,
                      const int* __restrict__ slots, const int* __restrict__ past, long tokens, int C, int R, int CS, int QR) {
  const int lane = threadIdx.x & 31;
  const long unit = (long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int units = dq ? 2 : 1;
  if (unit >= tokens * units) return;            // warps are independent
  const long tok = units == 2 ? unit >> 1 : unit;
  if (units == 2 && (unit & 1)) {
    const T* src = dq + tok * lddq;
    const float r = row_rms<T, VEC>(src, QR, eps, lane);
    T* dst = cq + tok * (long)QR;
    for (int i = lane * VEC; i < QR; i += 32 * VEC) {
      float f[VEC], w[VEC];
      Pack<T, VEC>::ld(src + i, f);
      Pack<T, VEC>::ld(wq + i, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) f[e] = f[e] * r * w[e];
      Pack<T, VEC>::st(dst + i, f);
    }
    return;
  }
  const int b = tok_seq[tok], p = past[b] + (int)(tok - seq_off[b]);
  T* row = pool + ((long)table[(long)slots[b] * max_pages + p / page_size] * page_size + p % page_size) * CS;
  T* out = lat ? lat + tok * (long)CS : nullptr;
  const T* src = dkv + tok * ldk;
  const float r = row_rms<T, VEC>(src, C, eps, lane);
  for (int i = lane * VEC; i < C; i += 32 * VEC) {
    float f[VEC], w[VEC];
    Pack<T, VEC>::ld(src + i, f);
    Pack<T, VEC>::ld(wkv + i, w);
#pragma unroll
    for (int e = 0; e < VEC; ++e) f[e] = f[e] * r * w[e];
    Pack<T, VEC>::st(row + i, f);
    if (out) Pack<T, VEC>::st(out + i, f);
  }
  for (int i = lane; i < R / 2; i += 32) {
    float c = 1.f, s = 0.f;
    if (i < half) { sincosf((float)p * freq[i], &s, &c); c *= mscale; s *= mscale; }
    cs[tok * (R / 2) + i] = make_float2(c, s);
    const float u = ldf(src + C + 2 * i), v = ldf(src + C + 2 * i + 1);
    const float a = u * c - v * s, d = v * c + u * s;
    stf(row + C + 2 * i, a); stf(row + C + 2 * i + 1, d);
    if (out) { stf(out + C + 2 * i, a); stf(out + C + 2 * i + 1, d); }
  }
  for (int i = C + R + lane; i < CS; i += 32) { stf(row + i, 0.f); if (out) stf(out + i, 0.f); }
}

// ext[e] = the cache row of position e - ext_off[b] of sequence b = ext_seq[e]; one unit U per thread (16 bytes where the rows allow it)
template <typename U>
__global__ void latent_pages_gather_kernel(const U* __restrict__ pool, const int* __restrict__ table, int max_pages, int page_size,
                                           const int* __restrict__ ext_seq, const int* __restrict__ ext_off, const int* __restrict__ slots,
                                           U* __restrict__ ext, long rows, int vecs) {
  const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= rows * vecs) return;
  const long e = i / vecs;
  const int c = (int)(i - e * vecs), b = ext_seq[e], p = (int)(e - ext_off[b]);
  ext[i] = pool[((long)table[(long)slots[b] * max_pages + p / page_size] * page_size + p % page_size) * vecs + c];
}

// ------------------------------------------------------------------------------------------------------------------
// Prompt attention on expanded keys and values, generic form: one warp per (row, head).  kv [ext rows, H*D keys | H*V values];
// lat [ext rows, ldl]: the shared key part sits at column C.  Row t sees the rows ext_off[b] .. ext_off[b] + position.
// ------------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void latent_prompt_kernel(const T* __restrict__ q, long ldq, const T* __restrict__ kv, long ldkv, const T* __restrict__ lat,
                                     long ldl, const float2* __restrict__ cs, const float* __restrict__ sink,
                                     const int* __restrict__ ext_off, const int* __restrict__ tok_seq, const int* __restrict__ seq_off,
                                     const int* __restrict__ past, T* __restrict__ y, long ldy, long tokens, int H, int D, int R, int V,
                                     int C, float scale) {
  extern __shared__ float sm[];
  const int wib = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long wid = (long)blockIdx.x * (blockDim.x >> 5) + wib;
  if (wid >= tokens * H) return;                 // warps are independent
  const long tok = wid / H;
  const int h = (int)(wid - tok * H), b = tok_seq[tok], n = past[b] + (int)(tok - seq_off[b]) + 1;
  const long e0 = ext_off[b];
  float* qs = sm + (long)wib * (D + R + V);
  float* acc = qs + D + R;
  const T* qr = q + tok * ldq + (long)h * (D + R);
  for (int i = lane; i < D; i += 32) qs[i] = ldf(qr + i);
  for (int i = lane; i < R / 2; i += 32) {
    const float2 t = cs[tok * (R / 2) + i];
    const float u = ldf(qr + D + 2 * i), v = ldf(qr + D + 2 * i + 1);
    qs[D + 2 * i] = u * t.x - v * t.y;
    qs[D + 2 * i + 1] = v * t.x + u * t.y;
  }
  for (int i = lane; i < V; i += 32) acc[i] = 0.f;
  __syncwarp();
  float m = -INFINITY, l = 0.f;
  for (int j0 = 0; j0 < n; j0 += 32) {
    const int j = j0 + lane;
    float s = -INFINITY;
    if (j < n) {
      const T* kr = kv + (e0 + j) * ldkv + (long)h * D;
      const T* rr = lat + (e0 + j) * ldl + C;
      float d = 0.f;
      for (int i = 0; i < D; ++i) d += qs[i] * ldf(kr + i);
      for (int i = 0; i < R; ++i) d += qs[D + i] * ldf(rr + i);
      s = d * scale;
    }
    const float mn = fmaxf(m, warp_max(s)), corr = expf(m - mn), pr = j < n ? expf(s - mn) : 0.f;
    l = l * corr + warp_sum(pr);
    m = mn;
    const int cnt = min(32, n - j0);
    for (int i = lane; i < (V + 31) / 32 * 32; i += 32) {
      float a = i < V ? acc[i] * corr : 0.f;
      const T* vr = kv + (e0 + j0) * ldkv + (long)H * D + (long)h * V + i;
      for (int k = 0; k < cnt; ++k) {
        const float pk = __shfl_sync(0xffffffffu, pr, k);
        if (i < V) a += pk * ldf(vr + k * ldkv);
      }
      if (i < V) acc[i] = a;
    }
  }
  float f = 1.f;
  if (sink) {
    const float mm = fmaxf(m, sink[h]);
    f = expf(m - mm);
    l = l * f + expf(sink[h] - mm);
  }
  f /= l;
  for (int i = lane; i < V; i += 32) stf(y + tok * ldy + (long)h * V + i, acc[i] * f);
}

// ------------------------------------------------------------------------------------------------------------------
// Tensor-core form of the prompt attention (bf16, mma.m16n8k16, ldmatrix, cp.async): a block of 4 warps owns 64 consecutive
// queries of one (sequence, head), 16 per warp, held as A fragments — the rotated part is turned in registers, where the
// interleaved pairs lie side by side — and walks the keys of the sequence 64 at a time through two shared-memory buffers.
// Key tile rows are [D | R | zeros] (DK = D + R padded), value rows [V | zeros] (VP).  D, R and V are multiples of 8.
// ------------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], const void* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ void cp_async16(void* smem, const void* gmem, bool full) {      // !full: 16 zero bytes
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(a), "l"(gmem), "r"(full ? 16 : 0));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

constexpr int PT_Q = 64, PT_K = 64;             // queries per block, keys per tile

template <int DK, int VP>
__global__ void __launch_bounds__(128, DK <= 128 && VP <= 128 ? 3 : 2)
latent_prompt_mma_kernel(const bf16* __restrict__ q, long ldq, const bf16* __restrict__ kv, long ldkv, const bf16* __restrict__ lat, long ldl,
                         const float2* __restrict__ cs, const float* __restrict__ sink, const int* __restrict__ ext_off,
                         const int* __restrict__ qt_seq, const int* __restrict__ qt_start, const int* __restrict__ seq_off,
                         const int* __restrict__ past, bf16* __restrict__ y, long ldy, int H, int D, int R, int V, int C, float scale) {
  constexpr int KS = DK + 8, VS = VP + 8, BUF = PT_K * (KS + VS);
  extern __shared__ __align__(16) unsigned char smraw[];
  bf16* const tiles = reinterpret_cast<bf16*>(smraw);                   // two buffers of [key tile | value tile]
  // the longest walks (last query tiles of a sequence) start first
  const int tile = gridDim.x - 1 - blockIdx.x;
  const int h = blockIdx.y, b = qt_seq[tile], t0 = qt_start[tile];
  const int n = seq_off[b + 1] - seq_off[b], p0 = past[b];
  const long tokbase = seq_off[b], e0 = ext_off[b];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int r0 = t0 + warp * 16 + gid, r1 = r0 + 8;                     // this lane's two query rows
  const int kend = p0 + min(t0 + PT_Q, n);                              // keys the block's last query sees
  const int ntiles = (kend + PT_K - 1) / PT_K;
  if (D + R < DK || V < VP) {                                           // padding columns: written once, never touched by the copies
    const int padk = (DK - D - R) / 8, padv = (VP - V) / 8;
    for (int c = threadIdx.x; c < 2 * PT_K * (padk + padv); c += 128) {
      const int row = c / (padk + padv), k = c - row * (padk + padv);
      bf16* kd = tiles + (row / PT_K) * BUF;
      bf16* dst = k < padk ? kd + (row % PT_K) * KS + D + R + k * 8 : kd + PT_K * KS + (row % PT_K) * VS + V + (k - padk) * 8;
      *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
    }
  }
  uint32_t qf[DK / 16][4];
#pragma unroll
  for (int kk = 0; kk < DK / 16; ++kk) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {                                       // e: rows r0 / r1, channels +0 / +8
      const int r = (e & 1) ? r1 : r0, c = kk * 16 + tig * 2 + (e >> 1) * 8;
      uint32_t v = 0u;
      if (r < n && c < D + R) {
        v = *reinterpret_cast<const uint32_t*>(q + (tokbase + r) * ldq + (long)h * (D + R) + c);
        if (c >= D) {
          const float2 t = cs[(tokbase + r) * (R / 2) + (c - D) / 2];
          const __nv_bfloat162 pr = *reinterpret_cast<const __nv_bfloat162*>(&v);
          const float u = __low2float(pr), w = __high2float(pr);
          v = pack_bf16(u * t.x - w * t.y, w * t.x + u * t.y);
        }
      }
      qf[kk][e] = v;
    }
  }
  float o[VP / 8][4];
#pragma unroll
  for (int j = 0; j < VP / 8; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;             // l: this lane's share of the row sums
  const int D8 = D / 8, K8 = (D + R) / 8, V8 = V / 8, per = K8 + V8;
  const bf16* const kbase = kv + (long)h * D;
  const bf16* const vbase = kv + (long)H * D + (long)h * V;
  const bf16* const rbase = lat + C;
  const int rstep = 128 / per, cstep = 128 - rstep * per, row_first = threadIdx.x / per, ch_first = threadIdx.x - row_first * per;
  auto prefetch = [&](int it) {
    bf16* kd = tiles + (it & 1) * BUF;
    bf16* vd = kd + PT_K * KS;
    int row = row_first, ch = ch_first;                                 // 16-byte column `ch` of key row `row`
    while (row < PT_K) {
      const int kp = it * PT_K + row;
      const bool ok = kp < kend;
      const long e = e0 + (ok ? kp : 0);
      if (ch < D8) cp_async16(kd + row * KS + ch * 8, kbase + e * ldkv + ch * 8, ok);
      else if (ch < K8) cp_async16(kd + row * KS + ch * 8, rbase + e * ldl + (ch - D8) * 8, ok);
      else cp_async16(vd + row * VS + (ch - K8) * 8, vbase + e * ldkv + (ch - K8) * 8, ok);
      row += rstep; ch += cstep;
      if (ch >= per) { ch -= per; ++row; }
    }
    cp_async_commit();
  };
  const int pw0 = p0 + t0 + warp * 16, pi0 = p0 + r0, pi1 = p0 + r1;    // positions: the warp's first query, this lane's rows
  prefetch(0);
  for (int it = 0; it < ntiles; ++it) {
    const int k0 = it * PT_K;
    if (it + 1 < ntiles) { prefetch(it + 1); cp_async_wait<1>(); } else { cp_async_wait<0>(); }
    __syncthreads();                                                    // every thread's part of tile `it` has landed
    const bf16* Ks = tiles + (it & 1) * BUF;
    const bf16* Vs = Ks + PT_K * KS;
    if (k0 <= pw0 + 15) {                                               // something in this tile for the warp's queries
      float sacc[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j) { sacc[j][0] = sacc[j][1] = sacc[j][2] = sacc[j][3] = 0.f; }
      const bf16* krow = Ks + ((lane >> 4) * 8 + (lane & 7)) * KS + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
          uint32_t bk[4];
          ldsm_x4(bk, krow + j * 8 * KS + kk * 16);
          mma_bf16(sacc[j], qf[kk], bk[0], bk[1]);
          mma_bf16(sacc[j + 1], qf[kk], bk[2], bk[3]);
        }
      }
      float mx0 = -INFINITY, mx1 = -INFINITY;
      const bool whole = k0 + PT_K - 1 <= pw0;                          // every query of the warp sees the whole tile
#pragma unroll
      for (int j = 0; j < 8; ++j) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          float sv = sacc[j][c] * scale;
          if (!whole && k0 + j * 8 + tig * 2 + (c & 1) > (c < 2 ? pi0 : pi1)) sv = -INFINITY;
          sacc[j][c] = sv;
          if (c < 2) mx0 = fmaxf(mx0, sv); else mx1 = fmaxf(mx1, sv);
        }
      }
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1)); mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1)); mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
      const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);           // finite: key 0 is seen by every row from the first tile on
      const float c0 = __expf(m0 - mn0), c1 = __expf(m1 - mn1);
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float pv = __expf(sacc[j][c] - (c < 2 ? mn0 : mn1));
          sacc[j][c] = pv;
          if (c < 2) s0 += pv; else s1 += pv;
        }
      }
      l0 = l0 * c0 + s0; l1 = l1 * c1 + s1; m0 = mn0; m1 = mn1;
      if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {            // a row maximum moved
#pragma unroll
        for (int j = 0; j < VP / 8; ++j) { o[j][0] *= c0; o[j][1] *= c0; o[j][2] *= c1; o[j][3] *= c1; }
      }
#pragma unroll
      for (int k2 = 0; k2 < PT_K / 16; ++k2) {
        uint32_t a[4];
        a[0] = pack_bf16(sacc[2 * k2][0], sacc[2 * k2][1]); a[1] = pack_bf16(sacc[2 * k2][2], sacc[2 * k2][3]);
        a[2] = pack_bf16(sacc[2 * k2 + 1][0], sacc[2 * k2 + 1][1]); a[3] = pack_bf16(sacc[2 * k2 + 1][2], sacc[2 * k2 + 1][3]);
        const bf16* vrow = Vs + (k2 * 16 + (lane & 15)) * VS + (lane >> 4) * 8;
#pragma unroll
        for (int j = 0; j < VP / 8; j += 2) {
          uint32_t bv[4];
          ldsm_x4_t(bv, vrow + j * 8);
          mma_bf16(o[j], a, bv[0], bv[1]);
          mma_bf16(o[j + 1], a, bv[2], bv[3]);
        }
      }
    }
    __syncthreads();                                                    // all warps are done with this buffer
  }
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  float i0 = 1.f, i1 = 1.f;
  if (sink) {                                                           // an entry of the denominator without a key or a value
    const float sk = sink[h], mm0 = fmaxf(m0, sk), mm1 = fmaxf(m1, sk);
    i0 = expf(m0 - mm0); i1 = expf(m1 - mm1);
    l0 = l0 * i0 + expf(sk - mm0); l1 = l1 * i1 + expf(sk - mm1);
  }
  i0 /= l0; i1 /= l1;
#pragma unroll
  for (int j = 0; j < VP / 8; ++j) {
    const int col = j * 8 + tig * 2;
    if (col < V) {
      bf16* dst = y + (long)h * V + col;
      if (r0 < n) *reinterpret_cast<uint32_t*>(dst + (tokbase + r0) * ldy) = pack_bf16(o[j][0] * i0, o[j][1] * i0);
      if (r1 < n) *reinterpret_cast<uint32_t*>(dst + (tokbase + r1) * ldy) = pack_bf16(o[j][2] * i1, o[j][3] * i1);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------------
// Absorbed form, step 1: qa[t, h, :C] = sum_d q[t, h, d] W_uk[h*D + d, :], qa[t, h, C:C+R] = the rotated query part (fp32).
// Block (head, 64 channels, BT rows): the eight warps share the D rows of the head's matrix, two channels per lane.
// ------------------------------------------------------------------------------------------------------------------
template <typename T, int BT>
__global__ void __launch_bounds__(256)
latent_absorb_kernel(const T* __restrict__ q, long ldq, const T* __restrict__ wuk, const float2* __restrict__ cs, float* __restrict__ qa,
                     long rows, int H, int D, int R, int C) {
  extern __shared__ float sm[];
  float* qs = sm;                                // [BT][D]
  float* red = sm + BT * D;                      // [7][BT][64]
  const int h = blockIdx.x, c0 = blockIdx.y * 64, tid = threadIdx.x, grp = tid >> 5, lane = tid & 31, c = c0 + lane * 2;
  const long t0 = (long)blockIdx.z * BT;
  const int nt = (int)min((long)BT, rows - t0);
  const int CA = C + R;
  for (int i = tid; i < BT * D; i += 256) {
    const int r = i / D, d = i - r * D;
    qs[i] = r < nt ? ldf(q + (t0 + r) * ldq + (long)h * (D + R) + d) : 0.f;
  }
  if (blockIdx.y == 0) {
    for (int i = tid; i < nt * (R / 2); i += 256) {
      const int r = i / (R / 2), k = i - r * (R / 2);
      const float2 t = cs[(t0 + r) * (R / 2) + k];
      const T* src = q + (t0 + r) * ldq + (long)h * (D + R) + D + 2 * k;
      const float u = ldf(src), v = ldf(src + 1);
      float* dst = qa + ((t0 + r) * H + h) * CA + C + 2 * k;
      dst[0] = u * t.x - v * t.y;
      dst[1] = v * t.x + u * t.y;
    }
  }
  __syncthreads();
  const int per = (D + 7) / 8, d0 = grp * per, d1 = min(D, d0 + per);
  float a0[BT], a1[BT];
#pragma unroll
  for (int r = 0; r < BT; ++r) { a0[r] = a1[r] = 0.f; }
  if (c < C) {
    const bool two = c + 1 < C, wide = two && sizeof(T) == 2 && (C & 1) == 0 && (reinterpret_cast<uintptr_t>(wuk) & 3) == 0;
#pragma unroll 8
    for (int d = d0; d < d1; ++d) {
      const T* wr = wuk + ((long)h * D + d) * C + c;
      float w0, w1;
      if (wide) {
        const __nv_bfloat162 p = *reinterpret_cast<const __nv_bfloat162*>(wr);
        w0 = __low2float(p); w1 = __high2float(p);
      } else {
        w0 = ldf(wr); w1 = two ? ldf(wr + 1) : 0.f;
      }
#pragma unroll
      for (int r = 0; r < BT; ++r) { a0[r] += qs[r * D + d] * w0; a1[r] += qs[r * D + d] * w1; }
    }
  }
  if (grp) {
#pragma unroll
    for (int r = 0; r < BT; ++r) { float* dst = red + ((grp - 1) * BT + r) * 64 + lane * 2; dst[0] = a0[r]; dst[1] = a1[r]; }
  }
  __syncthreads();
  if (grp == 0 && c < C) {
#pragma unroll
    for (int r = 0; r < BT; ++r) {
      if (r < nt) {
        for (int g = 0; g < 7; ++g) { const float* src = red + (g * BT + r) * 64 + lane * 2; a0[r] += src[0]; a1[r] += src[1]; }
        float* dst = qa + ((t0 + r) * H + h) * CA + c;
        dst[0] = a0[r];
        if (c + 1 < C) dst[1] = a1[r];
      }
    }
  }
}

// the keys [kbeg, kend) of part `part` of `nparts` of the n keys that a row sees (whole tiles of `tile` keys)
__device__ __forceinline__ void part_range(int n, int part, int nparts, int tile, int& kbeg, int& kend) {
  int len = (n + nparts - 1) / nparts;
  len = (len + tile - 1) / tile * tile;
  kbeg = min(n, part * len);
  kend = min(n, kbeg + len);
}

// ------------------------------------------------------------------------------------------------------------------
// Absorbed form, step 2, generic: block (part, group of AG heads, row).  16 cache rows at a time in shared memory as fp32, the
// scores of every (head, key) pair by two neighbouring lanes, online softmax per head, a thread owns up to AC latent channels.
// Partial results: part [rows, H, nparts, C + 2] = (maximum, sum, unnormalised latent).
// ------------------------------------------------------------------------------------------------------------------
constexpr int AG = 8, AK = 16, AC = 8;          // heads per block, keys per tile, latent channels per thread (C <= 2048)

template <typename T>
__global__ void __launch_bounds__(256)
latent_absorbed_kernel(const float* __restrict__ qa, const T* __restrict__ pool, const int* __restrict__ table, int max_pages, int page_size,
                       const int* __restrict__ tok_seq, const int* __restrict__ seq_off, const int* __restrict__ slots,
                       const int* __restrict__ past, float* __restrict__ part, int nparts, int H, int C, int R, int CS, float scale) {
  extern __shared__ float sm[];
  const int CA = C + R, LS = CA + 1;
  float* qs = sm;                                // [AG][CA] scaled queries
  float* ks = qs + AG * CA;                      // [AK][LS]
  float* ps = ks + AK * LS;                      // [AG][AK] scores, then probabilities
  float* ms = ps + AG * AK;                      // [AG] running maximum
  float* lsum = ms + AG;                         // [AG] running sum
  float* corr = lsum + AG;                       // [AG] correction of this tile
  const int tid = threadIdx.x, h0 = blockIdx.y * AG, hg = min(AG, H - h0);
  const long row = blockIdx.z;
  const int b = tok_seq[row], n = past[b] + (int)(row - seq_off[b]) + 1;
  const long slot = slots[b];
  int kbeg, kend;
  part_range(n, blockIdx.x, nparts, AK, kbeg, kend);
  for (int i = tid; i < AG * CA; i += 256) qs[i] = i < hg * CA ? qa[(row * H + h0) * CA + i] * scale : 0.f;
  if (tid < AG) { ms[tid] = -INFINITY; lsum[tid] = 0.f; }
  float acc[AG][AC];
#pragma unroll
  for (int g = 0; g < AG; ++g)
#pragma unroll
    for (int j = 0; j < AC; ++j) acc[g][j] = 0.f;
  for (int k0 = kbeg; k0 < kend; k0 += AK) {
    __syncthreads();                             // the previous tile has been read
    for (int i = tid; i < AK * CA; i += 256) {
      const int j = i / CA, c = i - j * CA, kp = k0 + j;
      ks[j * LS + c] = kp < kend ? ldf(pool + ((long)table[slot * max_pages + kp / page_size] * page_size + kp % page_size) * CS + c) : 0.f;
    }
    __syncthreads();
    {
      const int g = tid >> 5, j = (tid & 31) >> 1;               // 8 heads x 16 keys, two lanes each
      const float* qr = qs + g * CA;
      const float* kr = ks + j * LS;
      float d = 0.f;
      for (int c = tid & 1; c < CA; c += 2) d += qr[c] * kr[c];
      d += __shfl_xor_sync(0xffffffffu, d, 1);
      const float s = k0 + j < kend ? d : -INFINITY;
      const float mo = ms[g], mn = fmaxf(mo, warp_max(s));       // a warp per head
      const float pr = expf(s - mn);
      const float sum = 0.5f * warp_sum(pr);                     // every key is held by two lanes
      if ((tid & 1) == 0) ps[g * AK + j] = pr;
      __syncwarp();
      if ((tid & 31) == 0) { const float cr = expf(mo - mn); corr[g] = cr; lsum[g] = lsum[g] * cr + sum; ms[g] = mn; }
    }
    __syncthreads();
#pragma unroll
    for (int jc = 0; jc < AC; ++jc) {
      const int c = tid + jc * 256;
      if (c < C) {
#pragma unroll
        for (int g = 0; g < AG; ++g) acc[g][jc] *= corr[g];
        for (int j = 0; j < AK; ++j) {
          const float kvv = ks[j * LS + c];
#pragma unroll
          for (int g = 0; g < AG; ++g) acc[g][jc] += ps[g * AK + j] * kvv;
        }
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int g = 0; g < AG; ++g) {
    if (g < hg) {
      float* dst = part + (((row * H + h0 + g) * nparts) + blockIdx.x) * (long)(C + 2);
      if (tid == 0) { dst[0] = ms[g]; dst[1] = lsum[g]; }
      if (kbeg < kend)
#pragma unroll
        for (int jc = 0; jc < AC; ++jc) { const int c = tid + jc * 256; if (c < C) dst[2 + c] = acc[g][jc]; }
    }
  }
}

// ------------------------------------------------------------------------------------------------------------------
// The same on the tensor cores (bf16 cache): block (part, group of 16 heads, row) of 8 warps, 64 cache rows per tile in shared
// memory (cp.async, one or two buffers).  The fp32 absorbed queries are kept as a sum of two bf16 matrices (value and rounding
// rest), so a score is exact to the cache's own rounding.
//   1  warp w: scores of its 8 keys for the 16 heads;   2  warp w: online softmax of heads 2w, 2w + 1;
//   3  warp w: O[16, its NT * 8 channels] <- O * correction + P K, O in registers.
// ------------------------------------------------------------------------------------------------------------------
constexpr int MK = 64, MH = 16;

template <int NT>
__global__ void __launch_bounds__(256, 1)
latent_absorbed_mma_kernel(const float* __restrict__ qa, const bf16* __restrict__ pool, const int* __restrict__ table, int max_pages,
                           int page_size, const int* __restrict__ tok_seq, const int* __restrict__ seq_off, const int* __restrict__ slots,
                           const int* __restrict__ past, float* __restrict__ part, int nparts, int nbuf, int H, int C, int R, int CS,
                           float scale) {
  extern __shared__ __align__(16) unsigned char smraw[];
  const int CA = C + R, KW = (CS + 31) / 32 * 32, LS = KW + 8;
  bf16* const Kt = reinterpret_cast<bf16*>(smraw);               // [nbuf][MK][LS]
  bf16* const Qh = Kt + nbuf * MK * LS;                          // [MH][LS] query, and its rounding rest
  bf16* const Ql = Qh + MH * LS;
  bf16* const Ps = Ql + MH * LS;                                 // [MH][MK + 8]
  float* const Ss = reinterpret_cast<float*>(Ps + MH * (MK + 8));   // [MH][MK + 1]
  float* const Cr = Ss + MH * (MK + 1);                          // [MH] correction of this tile
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;
  const int h0 = blockIdx.y * MH, hg = min(MH, H - h0);
  const long row = blockIdx.z;
  const int b = tok_seq[row], n = past[b] + (int)(row - seq_off[b]) + 1;
  const long slot = slots[b];
  int kbeg, kend;
  part_range(n, blockIdx.x, nparts, MK, kbeg, kend);
  if (kbeg >= kend) {                                            // nothing in this part: the whole block leaves
    if (tid < hg) { float* dst = part + (((row * H + h0 + tid) * nparts) + blockIdx.x) * (long)(C + 2); dst[0] = -INFINITY; dst[1] = 0.f; }
    return;
  }
  const int ntiles = (kend - kbeg + MK - 1) / MK, per = CS / 8;
  auto load = [&](int it) {
    bf16* dst = Kt + (nbuf == 2 ? (it & 1) : 0) * MK * LS;
    for (int j = warp; j < MK; j += 8) {                         // a warp per row: the page is looked up once
      const int kp = kbeg + it * MK + j;
      const bool ok = kp < kend;
      const bf16* src = pool;
      if (ok) src += ((long)table[slot * max_pages + kp / page_size] * page_size + kp % page_size) * CS;
      for (int c = lane; c < per; c += 32) cp_async16(dst + j * LS + c * 8, src + c * 8, ok);
    }
    cp_async_commit();
  };
  load(0);
  for (int i = tid; i < nbuf * MK * (KW - CS) / 8; i += 256) {   // padding columns of the tiles, written once
    const int pad = (KW - CS) / 8, r = i / pad;
    *reinterpret_cast<uint4*>(Kt + r * LS + CS + (i - r * pad) * 8) = make_uint4(0u, 0u, 0u, 0u);
  }
  for (int i = tid; i < MH * KW; i += 256) {
    const int g = i / KW, c = i - g * KW;
    const float v = (g < hg && c < CA) ? qa[(row * H + h0 + g) * CA + c] : 0.f;
    const bf16 hi = __float2bfloat16_rn(v);
    Qh[g * LS + c] = hi;
    Ql[g * LS + c] = __float2bfloat16_rn(v - __bfloat162float(hi));
  }
  float o[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
  float m2[2] = {-INFINITY, -INFINITY}, l2[2] = {0.f, 0.f};      // heads 2 * warp and 2 * warp + 1
  const int cw0 = warp * NT * 8;                                 // first channel of this warp
  for (int it = 0; it < ntiles; ++it) {
    if (nbuf == 2 && it + 1 < ntiles) { load(it + 1); cp_async_wait<1>(); } else { cp_async_wait<0>(); }
    __syncthreads();
    const bf16* T0 = Kt + (nbuf == 2 ? (it & 1) : 0) * MK * LS;
    // 1: scores of keys 8 * warp .. + 7
    {
      float s[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f; }
      const bf16* krow = T0 + (warp * 8 + (lane & 7)) * LS + (lane >> 3) * 8;
      const int arow = (lane & 7) + 8 * ((lane >> 3) & 1), acol = 8 * (lane >> 4);
      const bf16* ah = Qh + arow * LS + acol;
      const bf16* al = Ql + arow * LS + acol;
#pragma unroll 2
      for (int c = 0; c < KW; c += 32) {
        uint32_t bk[4], a[4];
        ldsm_x4(bk, krow + c);
        ldsm_x4(a, ah + c);      mma_bf16(s[0], a, bk[0], bk[1]);
        ldsm_x4(a, al + c);      mma_bf16(s[1], a, bk[0], bk[1]);
        ldsm_x4(a, ah + c + 16); mma_bf16(s[2], a, bk[2], bk[3]);
        ldsm_x4(a, al + c + 16); mma_bf16(s[3], a, bk[2], bk[3]);
      }
      const int col = warp * 8 + tig * 2;
      float* d0 = Ss + gid * (MK + 1) + col;
      float* d1 = Ss + (gid + 8) * (MK + 1) + col;
      d0[0] = (s[0][0] + s[1][0] + s[2][0] + s[3][0]) * scale; d0[1] = (s[0][1] + s[1][1] + s[2][1] + s[3][1]) * scale;
      d1[0] = (s[0][2] + s[1][2] + s[2][2] + s[3][2]) * scale; d1[1] = (s[0][3] + s[1][3] + s[2][3] + s[3][3]) * scale;
    }
    __syncthreads();
    // 2: online softmax
    {
      const int left = kend - (kbeg + it * MK);                  // keys of this tile
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int g = 2 * warp + e;
        const float* sr = Ss + g * (MK + 1);
        const float sa = lane < left ? sr[lane] : -INFINITY, sb = lane + 32 < left ? sr[lane + 32] : -INFINITY;
        const float mn = fmaxf(m2[e], warp_max(fmaxf(sa, sb)));
        const float pa = expf(sa - mn), pb = expf(sb - mn), cr = expf(m2[e] - mn);
        l2[e] = l2[e] * cr + warp_sum(pa + pb);
        m2[e] = mn;
        Ps[g * (MK + 8) + lane] = __float2bfloat16_rn(pa);
        Ps[g * (MK + 8) + lane + 32] = __float2bfloat16_rn(pb);
        if (lane == 0) Cr[g] = cr;
      }
    }
    __syncthreads();
    // 3: O <- O * correction + P K
    {
      const float ca = Cr[gid], cb = Cr[gid + 8];
#pragma unroll
      for (int j = 0; j < NT; ++j) { o[j][0] *= ca; o[j][1] *= ca; o[j][2] *= cb; o[j][3] *= cb; }
#pragma unroll
      for (int k2 = 0; k2 < MK / 16; ++k2) {
        uint32_t a[4];
        ldsm_x4(a, Ps + ((lane & 7) + 8 * ((lane >> 3) & 1)) * (MK + 8) + k2 * 16 + 8 * (lane >> 4));
        const bf16* vrow = T0 + (k2 * 16 + (lane & 15)) * LS + cw0 + (lane >> 4) * 8;
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
          if (cw0 + j * 8 < C) {                                 // warp-uniform; a pair that starts inside C stays inside the padded row
            uint32_t bv[4];
            ldsm_x4_t(bv, vrow + j * 8);
            mma_bf16(o[j], a, bv[0], bv[1]);
            mma_bf16(o[j + 1], a, bv[2], bv[3]);
          }
        }
      }
    }
    if (nbuf == 1 && it + 1 < ntiles) { __syncthreads(); load(it + 1); }
    else __syncthreads();                                        // everybody is done with this buffer and with P
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int g = 2 * warp + e;
    if (g < hg && lane == 0) { float* dst = part + (((row * H + h0 + g) * nparts) + blockIdx.x) * (long)(C + 2); dst[0] = m2[e]; dst[1] = l2[e]; }
  }
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    const int c = cw0 + j * 8 + tig * 2;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int g = gid + 8 * e;
      if (g < hg && c < C) {
        float* dst = part + (((row * H + h0 + g) * nparts) + blockIdx.x) * (long)(C + 2) + 2 + c;
        dst[0] = o[j][2 * e];
        if (c + 1 < C) dst[1] = o[j][2 * e + 1];
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------------------------
// Absorbed form, step 3: merge the parts of BT rows of one head (the sink joins the denominator) and apply the value
// up-projection, y[t, h*V + v] = sum_c W_uv[h*V + v, c] lat[t, c]; a warp takes four value channels per turn.  The parts that hold
// keys are the first ones of a row.
// ------------------------------------------------------------------------------------------------------------------
template <typename T, int BT>
__global__ void __launch_bounds__(256)
latent_value_kernel(const float* __restrict__ part, int nparts, const float* __restrict__ sink, const T* __restrict__ wuv, T* __restrict__ y,
                    long ldy, long rows, int H, int V, int C) {
  extern __shared__ __align__(16) float sm[];
  __shared__ int used_s[BT];
  const int CP = (C + 3) & ~3;
  float* lat = sm;                               // [BT][CP]
  float* wt = sm + BT * CP;                      // [BT][nparts] weight of every part
  const int h = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const long t0 = (long)blockIdx.y * BT;
  const int nt = (int)min((long)BT, rows - t0);
  const long step = C + 2;
  if (warp < nt) {
    const float* base = part + (((t0 + warp) * H + h) * nparts) * step;
    float M = sink ? sink[h] : -INFINITY;
    int used = 0;
    for (int s = lane; s < nparts; s += 32) {
      const float m = base[s * step];
      M = fmaxf(M, m);
      if (m != -INFINITY) used = s + 1;
    }
    M = warp_max(M);
#pragma unroll
    for (int mk = 16; mk > 0; mk >>= 1) used = max(used, __shfl_xor_sync(0xffffffffu, used, mk));
    float L = 0.f;
    for (int s = lane; s < nparts; s += 32) {
      const float w = expf(base[s * step] - M);  // an empty part has maximum -inf: weight 0
      wt[warp * nparts + s] = w;
      L += w * base[s * step + 1];
    }
    L = warp_sum(L) + (sink ? expf(sink[h] - M) : 0.f);
    for (int s = lane; s < nparts; s += 32) wt[warp * nparts + s] /= L;
    if (lane == 0) used_s[warp] = used;
  }
  __syncthreads();
  for (int i = tid; i < BT * CP; i += 256) {
    const int r = i / CP, c = i - r * CP;
    float a = 0.f;
    if (r < nt && c < C) {
      const float* base = part + (((t0 + r) * H + h) * nparts) * step + 2 + c;
      const int used = used_s[r];
#pragma unroll 8
      for (int s = 0; s < used; ++s) a += wt[r * nparts + s] * base[s * step];
    }
    lat[i] = a;
  }
  __syncthreads();
  constexpr int PV = sizeof(T) == 2 ? 8 : 4;
  const bool vec = C % PV == 0 && (reinterpret_cast<uintptr_t>(wuv) & 15) == 0;
  for (int v0 = (blockIdx.z * 8 + warp) * 4; v0 < V; v0 += 32 * gridDim.z) {
    const T* wr[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) wr[k] = wuv + ((long)h * V + min(v0 + k, V - 1)) * C;
    float acc[4][BT];
#pragma unroll
    for (int k = 0; k < 4; ++k)
#pragma unroll
      for (int r = 0; r < BT; ++r) acc[k][r] = 0.f;
    if (vec) {
#pragma unroll 2
      for (int c = lane * PV; c < C; c += 32 * PV) {
        float w[4][PV];
#pragma unroll
        for (int k = 0; k < 4; ++k) Pack<T, PV>::ld(wr[k] + c, w[k]);
#pragma unroll
        for (int r = 0; r < BT; ++r) {
#pragma unroll
          for (int e = 0; e < PV; e += 4) {
            const float4 x = *reinterpret_cast<const float4*>(lat + r * CP + c + e);
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[k][r] += w[k][e] * x.x + w[k][e + 1] * x.y + w[k][e + 2] * x.z + w[k][e + 3] * x.w;
          }
        }
      }
    } else {
      for (int c = lane; c < C; c += 32) {
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float w = ldf(wr[k] + c);
#pragma unroll
          for (int r = 0; r < BT; ++r) acc[k][r] += w * lat[r * CP + c];
        }
      }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
#pragma unroll
      for (int r = 0; r < BT; ++r) {
        const float a = warp_sum(acc[k][r]);
        if (lane == 0 && r < nt && v0 + k < V) stf(y + (t0 + r) * ldy + (long)h * V + v0 + k, a);
      }
    }
  }
}

template <typename K> inline void allow_smem(K kernel, size_t bytes) {
  if (bytes > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}
inline size_t absorbed_mma_smem(int CS, int nbuf) {
  const size_t LS = (size_t)(CS + 31) / 32 * 32 + 8;
  return (size_t)nbuf * MK * LS * 2 + 2 * MH * LS * 2 + (size_t)MH * (MK + 8) * 2 + (size_t)MH * (MK + 1) * 4 + MH * 4;
}
}  // namespace

// ====================================================================================================================
// launchers (C ABI; return 0, a CUDA error code, or -1 for sizes a kernel is not built for)
// ====================================================================================================================
#define LAUNCH_END() do { cudaError_t e_ = cudaGetLastError(); return e_ == cudaSuccess ? 0 : (int)e_; } while (0)

extern "C" {

int lbl_latent_prepare(const void* dkv, long ldk, const void* dq, long lddq, const void* wkv, const void* wq, const float* freq, int half,
                       float mscale, float eps, void* pool, const int* table, int max_pages, int page_size, void* lat, void* cq, float* cs,
                       const int* tok_seq, const int* seq_off, const int* slots, const int* past, long tokens, int C, int R, int CS, int QR,
                       int dtype, cudaStream_t s) {
  if (tokens == 0) return 0;
  if (R % 2 != 0 || 2 * half > R || CS < C + R) return -1;
  const int warps = 4, pv = dtype ? 8 : 4;
  const unsigned grid = (unsigned)((tokens * (dq ? 2 : 1) + warps - 1) / warps);
  auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool v = C % pv == 0 && CS % pv == 0 && ldk % pv == 0 && al(dkv) && al(wkv) && al(pool) && (!lat || al(lat)) &&
                 (!dq || (QR % pv == 0 && lddq % pv == 0 && al(dq) && al(wq) && al(cq)));
#define LP(TT, VV) latent_prepare_kernel<TT, VV><<<grid, warps * 32, 0, s>>>((const TT*)dkv, ldk, (const TT*)dq, lddq, (const TT*)wkv, (const TT*)wq, freq, \
      half, mscale, eps, (TT*)pool, table, max_pages, page_size, (TT*)lat, (TT*)cq, (float2*)cs, tok_seq, seq_off, slots, past, tokens, C, R, CS, QR)
  if (dtype) { if (v) LP(bf16, 8); else LP(bf16, 1); } else { if (v) LP(float, 4); else LP(float, 1); }
#undef LP
  LAUNCH_END();
}

int lbl_latent_pages_gather(const void* pool, const int* table, int max_pages, int page_size, const int* ext_seq, const int* ext_off,
                            const int* slots, void* ext, long rows, int CS, int dtype, cudaStream_t s) {
  if (rows == 0) return 0;
  const long bytes = (long)CS * (dtype ? 2 : 4);
  const bool wide = bytes % 16 == 0 && ((uintptr_t)pool & 15) == 0 && ((uintptr_t)ext & 15) == 0;
  const int unit = wide ? 16 : (dtype ? 2 : 4), vecs = (int)(bytes / unit);
  const unsigned grid = (unsigned)((rows * vecs + 255) / 256);
#define PGA(U) latent_pages_gather_kernel<U><<<grid, 256, 0, s>>>((const U*)pool, table, max_pages, page_size, ext_seq, ext_off, slots, (U*)ext, rows, vecs)
  if (unit == 16) PGA(uint4); else if (unit == 2) PGA(uint16_t); else PGA(uint32_t);
#undef PGA
  LAUNCH_END();
}

int lbl_latent_prompt(const void* q, long ldq, const void* kv, long ldkv, const void* lat, long ldl, const float* cs, const float* sink,
                      const int* ext_off, const int* tok_seq, const int* seq_off, const int* past, void* y, long ldy, long tokens, int H,
                      int D, int R, int V, int C, float scale, int dtype, cudaStream_t s) {
  if (tokens == 0) return 0;
  const int warps = 4;
  const size_t smem = (size_t)warps * (D + R + V) * sizeof(float);
  if (smem > 200 * 1024) return -1;
  const unsigned grid = (unsigned)((tokens * H + warps - 1) / warps);
#define PG(TT) { allow_smem(latent_prompt_kernel<TT>, smem); \
    latent_prompt_kernel<TT><<<grid, warps * 32, smem, s>>>((const TT*)q, ldq, (const TT*)kv, ldkv, (const TT*)lat, ldl, (const float2*)cs, sink, \
        ext_off, tok_seq, seq_off, past, (TT*)y, ldy, tokens, H, D, R, V, C, scale); }
  if (dtype) PG(bf16) else PG(float)
#undef PG
  LAUNCH_END();
}

// bf16; D, R, V multiples of 8, D + R <= 256, V <= 256 (-1 otherwise)
int lbl_latent_prompt_mma(const void* q, long ldq, const void* kv, long ldkv, const void* lat, long ldl, const float* cs, const float* sink,
                          const int* ext_off, const int* qt_seq, const int* qt_start, int ntiles, const int* seq_off, const int* past, void* y,
                          long ldy, int H, int D, int R, int V, int C, float scale, cudaStream_t s) {
  if (ntiles == 0) return 0;
  if (D % 8 || R % 8 || V % 8 || C % 8 || D + R > 256 || V > 256 || ldq % 2 || ldkv % 8 || ldl % 8 || ldy % 2 || ((uintptr_t)q & 3) ||
      ((uintptr_t)kv & 15) || ((uintptr_t)lat & 15) || ((uintptr_t)y & 3) || ((uintptr_t)cs & 7)) return -1;
  const int dk = D + R <= 64 ? 64 : (D + R <= 96 ? 96 : (D + R <= 128 ? 128 : (D + R <= 192 ? 192 : 256)));
  const int vp = V <= 32 ? 32 : (V <= 64 ? 64 : (V <= 128 ? 128 : 256));
  const size_t smem = (size_t)2 * PT_K * (dk + 8 + vp + 8) * sizeof(bf16);
  const dim3 grid((unsigned)ntiles, (unsigned)H);
#define PM(DK_, VP_) { allow_smem(latent_prompt_mma_kernel<DK_, VP_>, smem); \
    latent_prompt_mma_kernel<DK_, VP_><<<grid, 128, smem, s>>>((const bf16*)q, ldq, (const bf16*)kv, ldkv, (const bf16*)lat, ldl, (const float2*)cs, \
        sink, ext_off, qt_seq, qt_start, seq_off, past, (bf16*)y, ldy, H, D, R, V, C, scale); }
#define PMV(DK_) { if (vp == 32) PM(DK_, 32) else if (vp == 64) PM(DK_, 64) else if (vp == 128) PM(DK_, 128) else PM(DK_, 256) }
  if (dk == 64) PMV(64) else if (dk == 96) PMV(96) else if (dk == 128) PMV(128) else if (dk == 192) PMV(192) else PMV(256)
#undef PMV
#undef PM
  LAUNCH_END();
}

int lbl_latent_absorb(const void* q, long ldq, const void* wuk, const float* cs, float* qa, long rows, int H, int D, int R, int C, int dtype,
                      cudaStream_t s) {
  if (rows == 0) return 0;
  const int bt = rows >= 8 ? 8 : (rows >= 3 ? 4 : (rows == 2 ? 2 : 1));
  const size_t smem = ((size_t)bt * D + 7 * (size_t)bt * 64) * sizeof(float);
  if (smem > 200 * 1024 || rows / bt > 60000) return -1;
  const dim3 grid((unsigned)H, (unsigned)((C + 63) / 64), (unsigned)((rows + bt - 1) / bt));
#define AB(TT, B_) { allow_smem(latent_absorb_kernel<TT, B_>, smem); \
    latent_absorb_kernel<TT, B_><<<grid, 256, smem, s>>>((const TT*)q, ldq, (const TT*)wuk, (const float2*)cs, qa, rows, H, D, R, C); }
#define ABT(TT) { if (bt == 8) AB(TT, 8) else if (bt == 4) AB(TT, 4) else if (bt == 2) AB(TT, 2) else AB(TT, 1) }
  if (dtype) ABT(bf16) else ABT(float)
#undef ABT
#undef AB
  LAUNCH_END();
}

// whether the tensor-core form takes these sizes (bf16 rows of CS channels)
int lbl_latent_absorbed_mma_ok(int C, int R, int CS) {
  return CS % 8 == 0 && C <= 1024 && CS >= C + R && absorbed_mma_smem(CS, 1) <= 220 * 1024;
}

// mma: 0 generic, 1 tensor cores (bf16)
int lbl_latent_absorbed(const float* qa, const void* pool, const int* table, int max_pages, int page_size, const int* tok_seq,
                        const int* seq_off, const int* slots, const int* past, float* part, int nparts, long rows, int H, int C, int R, int CS,
                        float scale, int mma, int dtype, cudaStream_t s) {
  if (rows == 0) return 0;
  if (rows > 60000 || nparts < 1) return -1;
  if (mma) {
    if (!dtype || !lbl_latent_absorbed_mma_ok(C, R, CS) || ((uintptr_t)pool & 15) != 0) return -1;
    const int nbuf = absorbed_mma_smem(CS, 2) <= 220 * 1024 ? 2 : 1;
    const size_t smem = absorbed_mma_smem(CS, nbuf);
    const dim3 grid((unsigned)nparts, (unsigned)((H + MH - 1) / MH), (unsigned)rows);
#define AM(NT_) { allow_smem(latent_absorbed_mma_kernel<NT_>, smem); \
    latent_absorbed_mma_kernel<NT_><<<grid, 256, smem, s>>>(qa, (const bf16*)pool, table, max_pages, page_size, tok_seq, seq_off, slots, past, part, \
        nparts, nbuf, H, C, R, CS, scale); }
    if (C <= 128) AM(2) else if (C <= 256) AM(4) else if (C <= 512) AM(8) else AM(16)
#undef AM
    LAUNCH_END();
  }
  const size_t smem = ((size_t)AG * (C + R) + (size_t)AK * (C + R + 1) + AG * AK + 3 * AG) * sizeof(float);
  if (C > AC * 256 || smem > 220 * 1024) return -1;
  const dim3 grid((unsigned)nparts, (unsigned)((H + AG - 1) / AG), (unsigned)rows);
#define AGK(TT) { allow_smem(latent_absorbed_kernel<TT>, smem); \
    latent_absorbed_kernel<TT><<<grid, 256, smem, s>>>(qa, (const TT*)pool, table, max_pages, page_size, tok_seq, seq_off, slots, past, part, nparts, H, \
        C, R, CS, scale); }
  if (dtype) AGK(bf16) else AGK(float)
#undef AGK
  LAUNCH_END();
}

int lbl_latent_value(const float* part, int nparts, const float* sink, const void* wuv, void* y, long ldy, long rows, int H, int V, int C,
                     int dtype, cudaStream_t s) {
  if (rows == 0) return 0;
  const int bt = rows * H >= 2048 ? 4 : 1;
  const size_t smem = ((size_t)bt * (C + 4) + (size_t)bt * nparts) * sizeof(float);
  const long groups = (rows + bt - 1) / bt;
  if (smem > 200 * 1024 || groups > 60000) return -1;
  int vz = (int)(148 / (groups * H)); if (vz > (V + 31) / 32) vz = (V + 31) / 32; if (vz < 1) vz = 1;
  const dim3 grid((unsigned)H, (unsigned)groups, (unsigned)vz);
#define LV(TT, B_) { allow_smem(latent_value_kernel<TT, B_>, smem); \
    latent_value_kernel<TT, B_><<<grid, 256, smem, s>>>(part, nparts, sink, (const TT*)wuv, (TT*)y, ldy, rows, H, V, C); }
  if (dtype) { if (bt == 4) LV(bf16, 4) else LV(bf16, 1) } else { if (bt == 4) LV(float, 4) else LV(float, 1) }
#undef LV
  LAUNCH_END();
}

}  // extern "C"
