// torch.ops.libai_b200_kv.latent_* : argument-checking wrappers around the launchers of latent_mixers.cu (attention on paged
// low-rank latents with a shared rotated key part), registered into the library of kv_bindings.cpp.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/library.h>
#include <torch/torch.h>

extern "C" {
int lbl_latent_prepare(const void* dkv, long ldk, const void* dq, long lddq, const void* wkv, const void* wq, const float* freq, int half,
                       float mscale, float eps, void* pool, const int* table, int max_pages, int page_size, void* lat, void* cq, float* cs,
                       const int* tok_seq, const int* seq_off, const int* slots, const int* past, long tokens, int C, int R, int CS, int QR,
                       int dtype, cudaStream_t s);
int lbl_latent_pages_gather(const void* pool, const int* table, int max_pages, int page_size, const int* ext_seq, const int* ext_off,
                            const int* slots, void* ext, long rows, int CS, int dtype, cudaStream_t s);
int lbl_latent_prompt(const void* q, long ldq, const void* kv, long ldkv, const void* lat, long ldl, const float* cs, const float* sink,
                      const int* ext_off, const int* tok_seq, const int* seq_off, const int* past, void* y, long ldy, long tokens, int H,
                      int D, int R, int V, int C, float scale, int dtype, cudaStream_t s);
int lbl_latent_prompt_mma(const void* q, long ldq, const void* kv, long ldkv, const void* lat, long ldl, const float* cs, const float* sink,
                          const int* ext_off, const int* qt_seq, const int* qt_start, int ntiles, const int* seq_off, const int* past, void* y,
                          long ldy, int H, int D, int R, int V, int C, float scale, cudaStream_t s);
int lbl_latent_absorb(const void* q, long ldq, const void* wuk, const float* cs, float* qa, long rows, int H, int D, int R, int C, int dtype,
                      cudaStream_t s);
int lbl_latent_absorbed_mma_ok(int C, int R, int CS);
int lbl_latent_absorbed(const float* qa, const void* pool, const int* table, int max_pages, int page_size, const int* tok_seq,
                        const int* seq_off, const int* slots, const int* past, float* part, int nparts, long rows, int H, int C, int R, int CS,
                        float scale, int mma, int dtype, cudaStream_t s);
int lbl_latent_value(const float* part, int nparts, const float* sink, const void* wuv, void* y, long ldy, long rows, int H, int V, int C,
                     int dtype, cudaStream_t s);
}

namespace {
using at::Tensor;
using OptT = c10::optional<Tensor>;

cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }
void check(int err, const char* what) {
  TORCH_CHECK(err == 0, what, err < 0 ? ": unsupported sizes" : ": CUDA error ", err < 0 ? "" : cudaGetErrorString((cudaError_t)err));
}
int code(const Tensor& t) {
  TORCH_CHECK(t.scalar_type() == at::kFloat || t.scalar_type() == at::kBFloat16, "float32 or bfloat16 expected");
  return t.scalar_type() == at::kFloat ? 0 : 1;
}
bool has(const OptT& t) { return t.has_value() && t->defined(); }
void rows2d(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.dim() == 2 && (t.size(1) == 1 || t.stride(1) == 1), name, ": 2-D CUDA tensor with unit column stride expected");
}
const int* meta(const Tensor& t) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kInt && t.is_contiguous(), "int32 CUDA metadata expected");
  return t.data_ptr<int>();
}
const float* f32(const Tensor& t, int64_t n, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous() && t.numel() == n, name, ": contiguous fp32 tensor of ", n, " numbers expected");
  return t.data_ptr<float>();
}
const float* sink_of(const OptT& sink, int64_t H) { return has(sink) ? f32(*sink, H, "latent attention sink") : nullptr; }
void vec(const Tensor& t, int64_t n, int dtype, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.is_contiguous() && t.numel() == n && code(t) == dtype, name, ": contiguous vector of the model's dtype expected");
}
void pool_shape(const Tensor& pool, const Tensor& table, int64_t channels, int dtype) {
  TORCH_CHECK(pool.is_cuda() && pool.is_contiguous() && pool.dim() == 3 && pool.size(2) >= channels && code(pool) == dtype, "latent attention: pool [pages, page_size, CS >= C + R]");
  TORCH_CHECK(table.dim() == 2, "latent attention: table [slots, max_pages]");
}

// dkv [tokens, C + R] and dq [tokens, QR]: column slices of projections.  Writes the page rows, cs [tokens, R / 2, 2], and — when
// given — lat [tokens, CS] (the same rows, packed) and cq [tokens, QR]
void latent_prepare(const Tensor& dkv, const OptT& dq, const Tensor& wkv, const OptT& wq, const Tensor& freq, double mscale, double eps,
                    Tensor pool, const Tensor& table, const OptT& lat, const OptT& cq, Tensor cs, const Tensor& tok_seq,
                    const Tensor& seq_off, const Tensor& slots, const Tensor& past, int64_t C, int64_t R) {
  rows2d(dkv, "latent_prepare dkv");
  const int dtype = code(dkv);
  const int64_t tokens = dkv.size(0), CS = pool.size(2);
  TORCH_CHECK(dkv.size(1) == C + R && R % 2 == 0, "latent_prepare: dkv [tokens, C + R], R even");
  vec(wkv, C, dtype, "latent_prepare latent norm");
  pool_shape(pool, table, C + R, dtype);
  TORCH_CHECK(freq.is_cuda() && freq.scalar_type() == at::kFloat && freq.is_contiguous() && 2 * freq.numel() <= R, "latent_prepare: freq fp32, at most R / 2");
  f32(cs, tokens * R, "latent_prepare cs");
  const void* dqp = nullptr; const void* wqp = nullptr; void* cqp = nullptr; long lddq = 0; int64_t QR = 0;
  if (has(dq)) {
    rows2d(*dq, "latent_prepare dq");
    QR = dq->size(1);
    TORCH_CHECK(dq->size(0) == tokens && code(*dq) == dtype && has(wq) && has(cq), "latent_prepare: dq with its norm and output");
    vec(*wq, QR, dtype, "latent_prepare query norm");
    TORCH_CHECK(cq->is_cuda() && cq->is_contiguous() && cq->dim() == 2 && cq->size(0) == tokens && cq->size(1) == QR && code(*cq) == dtype, "latent_prepare: cq [tokens, QR]");
    dqp = dq->data_ptr(); wqp = wq->data_ptr(); cqp = cq->data_ptr(); lddq = dq->stride(0);
  }
  void* lp = nullptr;
  if (has(lat)) {
    TORCH_CHECK(lat->is_cuda() && lat->is_contiguous() && lat->dim() == 2 && lat->size(0) == tokens && lat->size(1) == CS && code(*lat) == dtype, "latent_prepare: lat [tokens, CS]");
    lp = lat->data_ptr();
  }
  c10::cuda::CUDAGuard guard(dkv.device());
  check(lbl_latent_prepare(dkv.data_ptr(), dkv.stride(0), dqp, lddq, wkv.data_ptr(), wqp, freq.data_ptr<float>(), (int)freq.numel(), (float)mscale,
                           (float)eps, pool.data_ptr(), meta(table), (int)table.size(1), (int)pool.size(1), lp, cqp, cs.data_ptr<float>(),
                           meta(tok_seq), meta(seq_off), meta(slots), meta(past), tokens, (int)C, (int)R, (int)CS, (int)QR, dtype, cur_stream()),
        "latent_prepare");
}

void latent_pages_gather(const Tensor& pool, const Tensor& table, const Tensor& ext_seq, const Tensor& ext_off, const Tensor& slots, Tensor ext) {
  const int dtype = code(pool);
  pool_shape(pool, table, 1, dtype);
  TORCH_CHECK(ext.is_cuda() && ext.is_contiguous() && ext.dim() == 2 && ext.size(1) == pool.size(2) && code(ext) == dtype && ext_seq.numel() == ext.size(0),
              "latent_pages_gather: ext [rows, CS] and the sequence of every row");
  c10::cuda::CUDAGuard guard(pool.device());
  check(lbl_latent_pages_gather(pool.data_ptr(), meta(table), (int)table.size(1), (int)pool.size(1), meta(ext_seq), meta(ext_off), meta(slots),
                                ext.data_ptr(), ext.size(0), (int)pool.size(2), dtype, cur_stream()), "latent_pages_gather");
}

// q [tokens, H*(D+R)] unrotated; kv [rows, H*D + H*V]; lat [rows, >= C + R].  With query tiles (qt_seq, qt_start: 64 queries each) the
// tensor-core kernel
void latent_prompt(const Tensor& q, const Tensor& kv, const Tensor& lat, const Tensor& cs, const OptT& sink, const Tensor& ext_off,
                   const Tensor& tok_seq, const Tensor& seq_off, const Tensor& past, const OptT& qt_seq, const OptT& qt_start, Tensor y,
                   int64_t H, int64_t D, int64_t R, int64_t V, int64_t C, double scale) {
  rows2d(q, "latent_prompt q"); rows2d(kv, "latent_prompt kv"); rows2d(lat, "latent_prompt lat"); rows2d(y, "latent_prompt y");
  const int dtype = code(q);
  const int64_t tokens = q.size(0);
  TORCH_CHECK(q.size(1) == H * (D + R) && kv.size(1) == H * (D + V) && lat.size(1) >= C + R && lat.size(0) == kv.size(0) && y.size(0) == tokens &&
              y.size(1) == H * V && code(kv) == dtype && code(lat) == dtype && code(y) == dtype, "latent_prompt: shapes");
  const float* sp = sink_of(sink, H);
  f32(cs, tokens * R, "latent_prompt cs");
  c10::cuda::CUDAGuard guard(q.device());
  if (has(qt_seq)) {
    TORCH_CHECK(dtype == 1 && has(qt_start) && qt_start->numel() == qt_seq->numel(), "latent_prompt: the tensor-core form is bf16 and needs its query tiles");
    check(lbl_latent_prompt_mma(q.data_ptr(), q.stride(0), kv.data_ptr(), kv.stride(0), lat.data_ptr(), lat.stride(0), cs.data_ptr<float>(), sp,
                                meta(ext_off), meta(*qt_seq), meta(*qt_start), (int)qt_seq->numel(), meta(seq_off), meta(past), y.data_ptr(),
                                y.stride(0), (int)H, (int)D, (int)R, (int)V, (int)C, (float)scale, cur_stream()), "latent_prompt (tensor cores)");
    return;
  }
  check(lbl_latent_prompt(q.data_ptr(), q.stride(0), kv.data_ptr(), kv.stride(0), lat.data_ptr(), lat.stride(0), cs.data_ptr<float>(), sp,
                          meta(ext_off), meta(tok_seq), meta(seq_off), meta(past), y.data_ptr(), y.stride(0), tokens, (int)H, (int)D, (int)R,
                          (int)V, (int)C, (float)scale, dtype, cur_stream()), "latent_prompt");
}

bool latent_absorbed_mma_ok(int64_t C, int64_t R, int64_t CS) { return lbl_latent_absorbed_mma_ok((int)C, (int)R, (int)CS) != 0; }

// q [rows, H*(D+R)] unrotated, wuk [H*D, C], wuv [H*V, C] -> y [rows, H*V]; every row attends over its sequence's cached rows
// 0 .. its own position, the keys cut into `nparts` parts
void latent_absorbed(const Tensor& q, const Tensor& wuk, const Tensor& wuv, const Tensor& cs, const OptT& sink, const Tensor& pool,
                     const Tensor& table, const Tensor& tok_seq, const Tensor& seq_off, const Tensor& slots, const Tensor& past, Tensor y,
                     int64_t H, int64_t D, int64_t R, int64_t V, int64_t C, double scale, int64_t nparts, bool mma) {
  rows2d(q, "latent_absorbed q"); rows2d(y, "latent_absorbed y");
  const int dtype = code(q);
  const int64_t rows = q.size(0);
  TORCH_CHECK(q.size(1) == H * (D + R) && y.size(0) == rows && y.size(1) == H * V && code(y) == dtype, "latent_absorbed: q [rows, H*(D+R)], y [rows, H*V]");
  TORCH_CHECK(wuk.is_cuda() && wuk.is_contiguous() && wuk.numel() == H * D * C && code(wuk) == dtype && wuv.is_cuda() && wuv.is_contiguous() &&
              wuv.numel() == H * V * C && code(wuv) == dtype, "latent_absorbed: up-projections [H*D, C] and [H*V, C]");
  pool_shape(pool, table, C + R, dtype);
  TORCH_CHECK(nparts >= 1 && tok_seq.numel() >= rows, "latent_absorbed: parts and row owners");
  const float* sp = sink_of(sink, H);
  f32(cs, rows * R, "latent_absorbed cs");
  c10::cuda::CUDAGuard guard(q.device());
  Tensor qa = at::empty({rows * H * (C + R)}, q.options().dtype(at::kFloat));
  Tensor part = at::empty({rows * H * nparts * (C + 2)}, q.options().dtype(at::kFloat));
  check(lbl_latent_absorb(q.data_ptr(), q.stride(0), wuk.data_ptr(), cs.data_ptr<float>(), qa.data_ptr<float>(), rows, (int)H, (int)D, (int)R, (int)C,
                          dtype, cur_stream()), "latent_absorb");
  check(lbl_latent_absorbed(qa.data_ptr<float>(), pool.data_ptr(), meta(table), (int)table.size(1), (int)pool.size(1), meta(tok_seq), meta(seq_off),
                            meta(slots), meta(past), part.data_ptr<float>(), (int)nparts, rows, (int)H, (int)C, (int)R, (int)pool.size(2), (float)scale,
                            mma ? 1 : 0, dtype, cur_stream()), "latent_absorbed");
  check(lbl_latent_value(part.data_ptr<float>(), (int)nparts, sp, wuv.data_ptr(), y.data_ptr(), y.stride(0), rows, (int)H, (int)V, (int)C, dtype,
                         cur_stream()), "latent_value");
}
}  // namespace

TORCH_LIBRARY_FRAGMENT(libai_b200_kv, m) {
  m.def("latent_prepare(Tensor dkv, Tensor? dq, Tensor wkv, Tensor? wq, Tensor freq, float mscale, float eps, Tensor(a!) pool, Tensor table, Tensor(b!)? lat, Tensor(c!)? cq, Tensor(d!) cs, Tensor tok_seq, Tensor seq_off, Tensor slots, Tensor past, int C, int R) -> ()", &latent_prepare);
  m.def("latent_pages_gather(Tensor pool, Tensor table, Tensor ext_seq, Tensor ext_off, Tensor slots, Tensor(a!) ext) -> ()", &latent_pages_gather);
  m.def("latent_prompt(Tensor q, Tensor kv, Tensor lat, Tensor cs, Tensor? sink, Tensor ext_off, Tensor tok_seq, Tensor seq_off, Tensor past, Tensor? qt_seq, Tensor? qt_start, Tensor(a!) y, int H, int D, int R, int V, int C, float scale) -> ()", &latent_prompt);
  m.def("latent_absorbed_mma_ok(int C, int R, int CS) -> bool", &latent_absorbed_mma_ok);
  m.def("latent_absorbed(Tensor q, Tensor wuk, Tensor wuv, Tensor cs, Tensor? sink, Tensor pool, Tensor table, Tensor tok_seq, Tensor seq_off, Tensor slots, Tensor past, Tensor(a!) y, int H, int D, int R, int V, int C, float scale, int nparts, bool mma) -> ()", &latent_absorbed);
}
