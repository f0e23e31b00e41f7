// Bindings of the layer-by-layer decoders' kernels: mixers.cu, latent_*.cu, linear_*.cu, window_*.cu, paged_attend.cu, experts_any.cu.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include "launch.h"

// A serving build (MB_SERVE_SUBSET) has the mixers it was asked for, any other build all of them.
#if !defined(MB_SERVE_SUBSET) || defined(MB_SERVE_LATENT)
#define MB_HAS_LATENT
#endif
#if !defined(MB_SERVE_SUBSET) || defined(MB_SERVE_ATTENTION)
#define MB_HAS_ATTENTION
#endif

namespace {

using OptTensor = c10::optional<at::Tensor>;

inline cudaStream_t cur_stream() {
  (void)cudaGetLastError();
  mb_count_launch(1);
  return at::cuda::getCurrentCUDAStream().stream();
}
inline const void* cptr(const OptTensor& t) { return t.has_value() && t->defined() ? t->data_ptr() : nullptr; }
inline void* mptr(const OptTensor& t) { return t.has_value() && t->defined() ? t->data_ptr() : nullptr; }
inline const int* iptr(const OptTensor& t) { return t.has_value() && t->defined() ? t->data_ptr<int>() : nullptr; }
inline const float* fptr(const OptTensor& t) { return t.has_value() && t->defined() ? t->data_ptr<float>() : nullptr; }
inline float* fmut(const OptTensor& t) { return t.has_value() && t->defined() ? t->data_ptr<float>() : nullptr; }
inline const long long* lptr(const at::Tensor& t) { return reinterpret_cast<const long long*>(t.data_ptr<int64_t>()); }
inline int f32(const at::Tensor& t) { return t.scalar_type() == at::kFloat; }
inline void check(int rc, const char* what) {
  if (rc == 0) return;
  char buf[256];
  snprintf(buf, sizeof(buf), "%s failed with code %d (%s)", what, rc,
           rc > 0 && rc < 1000 ? cudaGetErrorString(static_cast<cudaError_t>(rc)) : "launcher: sizes out of the kernel's range");
  throw std::runtime_error(buf);
}
void bigram_embedding(const at::Tensor& tok, const OptTensor& prev, const at::Tensor& embed, const OptTensor& table, int64_t buckets,
                      int64_t mul_prev, int64_t mul_cur, at::Tensor& x, const OptTensor& xb) {
  c10::cuda::CUDAGuard g(embed.device());
  check(mb_bigram_embedding(tok.data_ptr<int>(), iptr(prev), embed.data_ptr(), cptr(table), buckets, mul_prev, mul_cur, x.data_ptr<float>(),
                            mptr(xb), tok.numel(), embed.size(1), f32(embed), cur_stream()),
        "mb_bigram_embedding");
}

void output_norm(at::Tensor& x, const at::Tensor& y, const at::Tensor& nw, const at::Tensor& ls, const OptTensor& fw, at::Tensor& xb,
                 double eps) {
  c10::cuda::CUDAGuard g(x.device());
  check(mb_output_norm(x.data_ptr<float>(), y.data_ptr(), nw.data_ptr(), ls.data_ptr(), cptr(fw), xb.data_ptr(), x.size(0), x.size(1), eps, f32(y),
                       cur_stream()),
        "mb_output_norm");
}

void gemv_output_norm(const at::Tensor& x, const at::Tensor& y, const at::Tensor& nw, const at::Tensor& ls, double eps, const at::Tensor& w,
                      at::Tensor& out, at::Tensor& x_out, bool static_w) {
  c10::cuda::CUDAGuard g(x.device());
  check(mb_gemv_output_norm(x.data_ptr<float>(), y.data_ptr(), nw.data_ptr(), ls.data_ptr(), eps, w.data_ptr(), out.data_ptr(), out.stride(0),
                            x_out.data_ptr<float>(), x.size(0), w.size(0), x.size(1), static_w, cur_stream()),
        "mb_gemv_output_norm");
}

// rows of `in` [gate, up] and of `out` may be strided; rows (optional): device count of the rows in use
void clamped_glu(const at::Tensor& in, at::Tensor& out, double limit, double alpha, const OptTensor& rows) {
  c10::cuda::CUDAGuard g(in.device());
  TORCH_CHECK(in.stride(1) == 1 && out.stride(1) == 1 && in.size(1) >= 2 * out.size(1), "clamped_glu: rows of [gate, up]");
  check(mb_clamped_glu(in.data_ptr(), in.stride(0), out.data_ptr(), out.stride(0), out.size(0), out.size(1), limit, alpha, iptr(rows), f32(in),
                       cur_stream()),
        "mb_clamped_glu");
}

void sum_norm(const at::Tensor& x, const OptTensor& to, const OptTensor& y1, const OptTensor& y2, const OptTensor& rows, const OptTensor& weights,
              const OptTensor& dst, const OptTensor& extra, const OptTensor& nw, const OptTensor& h, double eps) {
  c10::cuda::CUDAGuard g(x.device());
  MbSumNorm p{};
  p.x = x.data_ptr<float>();
  p.to = fmut(to);
  p.y1 = cptr(y1);
  p.y2 = cptr(y2);
  p.rows = cptr(rows);
  p.weights = fptr(weights);
  p.dst = iptr(dst);
  p.extra = fptr(extra);
  p.nw = cptr(nw);
  p.h = mptr(h);
  p.T = x.size(0);
  p.D = x.size(1);
  p.k = p.weights != nullptr ? weights->size(1) : 0;
  p.eps = eps;
  for (const OptTensor* t : {&y1, &y2, &rows, &nw})
    TORCH_CHECK(!t->has_value() || !(*t)->defined() || (*t)->is_contiguous(), "sum_norm: contiguous rows");
  int is32 = 0;
  for (const OptTensor* t : {&nw, &y1, &y2, &rows})
    if (t->has_value() && (*t)->defined()) is32 = f32(**t);
  check(mb_sum_norm(p, is32, cur_stream()), "mb_sum_norm");
}

// x32 (with y1, y2, extra, norm_w) or plain rows x; W [N, K] → y, W2 [N2, K] → fp32 y2out
void gemv_sum_norm(const OptTensor& x32, const OptTensor& y1, const OptTensor& y2, const OptTensor& extra, const OptTensor& x, const OptTensor& norm_w,
                   double eps, const at::Tensor& W, at::Tensor& y, const OptTensor& W2, const OptTensor& bias2, const OptTensor& y2out,
                   const OptTensor& x_out, const OptTensor& xn_out, bool static_w) {
  c10::cuda::CUDAGuard g(W.device());
  const bool two = W2.has_value() && W2->defined();
  check(mb_gemv_sum_norm(fptr(x32), cptr(y1), cptr(y2), fptr(extra), cptr(x), cptr(norm_w), eps, W.data_ptr(), y.data_ptr(), y.stride(0), cptr(W2),
                         cptr(bias2), fmut(y2out), fmut(x_out), mptr(xn_out), y.size(0), W.size(0), two ? W2->size(0) : 0, W.size(1), static_w,
                         cur_stream()),
        "mb_gemv_sum_norm");
}

void gated_norm(const at::Tensor& o, const at::Tensor& w, const at::Tensor& gate, at::Tensor& out, double eps) {
  c10::cuda::CUDAGuard g(o.device());
  check(mb_gated_norm(o.data_ptr(), w.data_ptr(), gate.data_ptr(), gate.stride(0), out.data_ptr(), o.size(0), o.size(1), eps, f32(o), cur_stream()),
        "mb_gated_norm");
}

#ifdef MB_HAS_LATENT
inline MbLatent layout(const std::vector<int64_t>& v) {
  TORCH_CHECK(v.size() == 7, "latent layout has 7 sizes");
  return MbLatent{static_cast<int>(v[0]), static_cast<int>(v[1]), static_cast<int>(v[2]), static_cast<int>(v[3]),
                  static_cast<int>(v[4]), static_cast<int>(v[5]), static_cast<int>(v[6])};
}

void latent_prep(const at::Tensor& proj, const at::Tensor& positions, const at::Tensor& slots, const at::Tensor& freq, double magnitude,
                 const OptTensor& kv_norm, double eps, at::Tensor& cache, const OptTensor& q_abs, const OptTensor& q_full, int64_t t_long,
                 int64_t q_nope, int64_t q_width, const std::vector<int64_t>& lay) {
  c10::cuda::CUDAGuard g(proj.device());
  check(mb_latent_prep(proj.data_ptr(), proj.stride(0), positions.data_ptr<int>(), lptr(slots), freq.data_ptr<double>(), magnitude, cptr(kv_norm),
                       eps, cache.data_ptr(), mptr(q_abs), mptr(q_full), proj.size(0), t_long, q_nope, q_width, layout(lay), f32(proj),
                       cur_stream()),
        "mb_latent_prep");
}

// x [T, H, K] (any strides of T and H), w [H, N, K] (w_nk) or [H, K, N], y [T, H, N] (any strides of T and H)
void head_linear(const at::Tensor& x, const at::Tensor& w, bool w_nk, at::Tensor& y) {
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(x.stride(2) == 1 && y.stride(2) == 1 && w.is_contiguous(), "head_linear: innermost dimension must be contiguous");
  check(mb_head_linear(x.data_ptr(), x.stride(0), x.stride(1), w.data_ptr(), w_nk, y.data_ptr(), y.stride(0), y.stride(1), x.size(0), x.size(1),
                       y.size(2), x.size(2), f32(x), cur_stream()),
        "mb_head_linear");
}

void latent_attend(const at::Tensor& q, const at::Tensor& cache, const at::Tensor& block_table, const OptTensor& token_seq,
                   const at::Tensor& positions, const at::Tensor& slots, const OptTensor& sink, at::Tensor& out, double scale, int64_t window,
                   const std::vector<int64_t>& lay) {
  c10::cuda::CUDAGuard g(q.device());
  check(mb_latent_attend(q.data_ptr(), cache.data_ptr(), block_table.data_ptr<int>(), block_table.size(1), cache.size(1), iptr(token_seq),
                         positions.data_ptr<int>(), lptr(slots), cptr(sink), out.data_ptr(), q.size(0), scale, window, layout(lay), f32(q),
                         cur_stream()),
        "mb_latent_attend");
}

void latent_gather(const at::Tensor& cache, const at::Tensor& block_table, const at::Tensor& cu_k, const at::Tensor& base, at::Tensor& out) {
  c10::cuda::CUDAGuard g(cache.device());
  check(mb_latent_gather(cache.data_ptr(), block_table.data_ptr<int>(), block_table.size(1), cache.size(1), cu_k.data_ptr<int>(),
                         base.data_ptr<int>(), out.data_ptr(), base.numel(), out.size(0), cache.size(2), cur_stream()),
        "mb_latent_gather");
}

void head_linear_mma(const at::Tensor& x, const at::Tensor& w, bool w_nk, at::Tensor& y) {
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(x.stride(2) == 1 && y.stride(2) == 1 && w.is_contiguous(), "head_linear_mma: innermost dimension must be contiguous");
  check(mb_head_linear_mma(x.data_ptr(), x.stride(0), x.stride(1), w.data_ptr(), w_nk, y.data_ptr(), y.stride(0), y.stride(1), x.size(0),
                           x.size(1), y.size(2), x.size(2), cur_stream()),
        "mb_head_linear_mma");
}

void latent_decode(const at::Tensor& q, const at::Tensor& cache, const at::Tensor& block_table, const OptTensor& token_seq,
                   const at::Tensor& positions, const at::Tensor& slots, const OptTensor& sink, at::Tensor& part_o, at::Tensor& part_ml,
                   at::Tensor& out, double scale, int64_t window, int64_t splits, const std::vector<int64_t>& lay, at::Tensor& err) {
  c10::cuda::CUDAGuard g(q.device());
  mb_count_launch(1);
  check(mb_latent_decode(q.data_ptr(), cache.data_ptr(), block_table.data_ptr<int>(), block_table.size(1), cache.size(1), iptr(token_seq),
                         positions.data_ptr<int>(), lptr(slots), cptr(sink), part_o.data_ptr<float>(), part_ml.data_ptr<float>(), out.data_ptr(),
                         q.size(0), scale, window, splits, cache.size(0), layout(lay), err.data_ptr<int>(), cur_stream()),
        "mb_latent_decode");
}

void latent_prefill(const at::Tensor& q, const at::Tensor& kv, const at::Tensor& lat, at::Tensor& o, const OptTensor& sink, const at::Tensor& cu_q,
                    const at::Tensor& cu_k, int64_t n_seq, int64_t max_q, double scale, int64_t window, const std::vector<int64_t>& lay,
                    at::Tensor& err) {
  c10::cuda::CUDAGuard g(q.device());
  check(mb_latent_prefill(q.data_ptr(), kv.data_ptr(), lat.data_ptr(), o.data_ptr(), cptr(sink), cu_q.data_ptr<int>(), cu_k.data_ptr<int>(), n_seq,
                          max_q, q.size(0), lat.size(0), scale, window, layout(lay), err.data_ptr<int>(), cur_stream()),
        "mb_latent_prefill");
}

void linear_state(const at::Tensor& proj, const at::Tensor& decay, at::Tensor& state, const at::Tensor& slots, const OptTensor& cu_q,
                  const at::Tensor& positions, at::Tensor& out) {
  c10::cuda::CUDAGuard g(proj.device());
  check(mb_linear_state(proj.data_ptr(), proj.stride(0), decay.data_ptr<float>(), state.data_ptr<float>(), slots.data_ptr<int>(), iptr(cu_q),
                        positions.data_ptr<int>(), out.data_ptr(), slots.numel(), state.size(1), state.size(2), state.size(3), f32(proj),
                        cur_stream()),
        "mb_linear_state");
}

void linear_chunk(const at::Tensor& proj, const at::Tensor& decay, at::Tensor& state, const at::Tensor& slots, const at::Tensor& positions,
                  const at::Tensor& segs, const at::Tensor& seq_segs, const OptTensor& seg_state, at::Tensor& out) {
  c10::cuda::CUDAGuard g(proj.device());
  const bool multi = seg_state.has_value() && seg_state->defined();
  if (multi) mb_count_launch(2);
  check(mb_linear_chunk(proj.data_ptr(), proj.stride(0), decay.data_ptr<float>(), state.data_ptr<float>(), slots.data_ptr<int>(),
                        positions.data_ptr<int>(), segs.data_ptr<int>(), seq_segs.data_ptr<int>(), multi ? seg_state->data_ptr<float>() : nullptr,
                        out.data_ptr(), seq_segs.numel() - 1, segs.size(0), state.size(1), state.size(2), state.size(3), cur_stream()),
        "mb_linear_chunk");
}
#endif  // MB_HAS_LATENT

#ifdef MB_HAS_ATTENTION
inline MbWindow window(const std::vector<int64_t>& v) {
  TORCH_CHECK(v.size() == 8, "a windowed attention layout has 8 sizes");
  return MbWindow{static_cast<int>(v[0]), static_cast<int>(v[1]), static_cast<int>(v[2]), static_cast<int>(v[3]),
                  static_cast<int>(v[4]), static_cast<int>(v[5]), static_cast<int>(v[6]), static_cast<int>(v[7])};
}

void window_prep(const at::Tensor& proj, const at::Tensor& positions, const at::Tensor& slots, const at::Tensor& freq, double magnitude,
                 const OptTensor& q_norm, const OptTensor& k_norm, double eps, at::Tensor& kc, at::Tensor& vc, at::Tensor& q,
                 const std::vector<int64_t>& lay, const OptTensor& logits, const OptTensor& weights, const OptTensor& index, const OptTensor& glu_in,
                 const OptTensor& glu_out, double limit, double alpha) {
  c10::cuda::CUDAGuard g(proj.device());
  MbAside a{};
  if (logits.has_value() && logits->defined()) {
    a.logits = logits->data_ptr<float>();
    a.weights = fmut(weights);
    a.index = index->data_ptr<int>();
    a.experts = logits->size(1);
    a.top = index->size(1);
    TORCH_CHECK(logits->is_contiguous(), "window_prep: contiguous logits");
  }
  if (glu_in.has_value() && glu_in->defined()) {
    a.glu_in = glu_in->data_ptr();
    a.glu_out = mptr(glu_out);
    a.glu_ld_in = glu_in->stride(0);
    a.glu_ld_out = glu_out->stride(0);
    a.ff = glu_out->size(1);
    a.limit = limit;
    a.alpha = alpha;
  }
  check(mb_window_prep(proj.data_ptr(), proj.stride(0), positions.data_ptr<int>(), lptr(slots), freq.data_ptr<double>(), magnitude, cptr(q_norm),
                       cptr(k_norm), eps, kc.data_ptr(), vc.data_ptr(), q.data_ptr(), proj.size(0), window(lay), a, f32(proj), cur_stream()),
        "mb_window_prep");
}

void window_decode(const at::Tensor& q, const at::Tensor& kc, const at::Tensor& vc, const at::Tensor& block_table, const OptTensor& token_seq,
                   const at::Tensor& positions, const at::Tensor& slots, const OptTensor& sink, at::Tensor& out, double scale, int64_t splits,
                   const std::vector<int64_t>& lay) {
  c10::cuda::CUDAGuard g(q.device());
  check(mb_window_decode(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), block_table.data_ptr<int>(), block_table.size(1), kc.size(1), iptr(token_seq),
                         positions.data_ptr<int>(), lptr(slots), cptr(sink), out.data_ptr(), out.stride(0), q.size(0), scale, splits, window(lay),
                         cur_stream()),
        "mb_window_decode");
}

void window_attend(const at::Tensor& q, const at::Tensor& kc, const at::Tensor& vc, const at::Tensor& block_table, const OptTensor& token_seq,
                   const at::Tensor& positions, const at::Tensor& slots, const OptTensor& sink, at::Tensor& out, double scale,
                   const std::vector<int64_t>& lay) {
  c10::cuda::CUDAGuard g(q.device());
  const MbWindow L = window(lay);
  MbAttend a{};
  a.heads = L.heads;
  a.group = L.heads / L.kv_heads;
  a.dk = L.dim;
  a.dv = L.vdim;
  a.q_head = L.q_pitch;
  a.q_row = static_cast<long long>(L.heads) * L.q_pitch;
  a.k_head = L.dim;
  a.k_row = static_cast<long long>(L.kv_heads) * L.dim;
  a.v_head = L.vdim;
  a.v_row = static_cast<long long>(L.kv_heads) * L.vdim;
  a.o_row = out.stride(0);
  a.window = L.window;
  a.keep = L.keep;
  a.scale = scale;
  check(mb_paged_attend(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), block_table.data_ptr<int>(), block_table.size(1), kc.size(1), iptr(token_seq),
                        positions.data_ptr<int>(), lptr(slots), cptr(sink), out.data_ptr(), q.size(0), a, f32(q), cur_stream()),
        "mb_paged_attend");
}

void window_prefill(const at::Tensor& q, const at::Tensor& kc, const at::Tensor& vc, at::Tensor& out, const OptTensor& sink, const at::Tensor& cu_q,
                    const at::Tensor& positions, const at::Tensor& block_table, int64_t n_seq, int64_t max_q, int64_t t_long, double scale,
                    const std::vector<int64_t>& lay, at::Tensor& err) {
  c10::cuda::CUDAGuard g(q.device());
  check(mb_window_prefill(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), out.data_ptr(), out.stride(0), cptr(sink), cu_q.data_ptr<int>(),
                          positions.data_ptr<int>(), block_table.data_ptr<int>(), block_table.size(1), kc.size(1), kc.size(0), n_seq, max_q, t_long,
                          scale, window(lay), err.data_ptr<int>(), cur_stream()),
        "mb_window_prefill");
}

void experts_any(const at::Tensor& x, const at::Tensor& w13, const at::Tensor& w2, const at::Tensor& index, const at::Tensor& weights, at::Tensor& act,
                 at::Tensor& out, double limit, double alpha) {
  c10::cuda::CUDAGuard g(x.device());
  mb_count_launch(1);
  check(mb_experts_any(x.data_ptr(), w13.data_ptr(), w2.data_ptr(), index.data_ptr<int>(), weights.data_ptr<float>(), act.data_ptr(), out.data_ptr(),
                       x.size(0), index.size(1), w13.size(0), x.size(1), w2.size(2), limit, alpha, f32(x), cur_stream()),
        "mb_experts_any");
}
#endif  // MB_HAS_ATTENTION

}  // namespace

void register_mixers(pybind11::module& m) {
  m.def("bigram_embedding", &bigram_embedding);
  m.def("output_norm", &output_norm);
  m.def("gemv_output_norm", &gemv_output_norm);
  m.def("clamped_glu", &clamped_glu, pybind11::arg("in"), pybind11::arg("out"), pybind11::arg("limit"), pybind11::arg("alpha"),
        pybind11::arg("rows") = pybind11::none());
  m.def("sum_norm", &sum_norm);
  m.def("gemv_sum_norm", &gemv_sum_norm);
  m.def("gated_norm", &gated_norm);
#ifdef MB_HAS_LATENT
  m.def("latent_prep", &latent_prep);
  m.def("head_linear", &head_linear);
  m.def("latent_attend", &latent_attend);
  m.def("latent_gather", &latent_gather);
  m.def("head_linear_mma", &head_linear_mma);
  m.def("latent_decode", &latent_decode);
  m.def("latent_prefill", &latent_prefill);
  m.def("linear_state", &linear_state);
  m.def("linear_chunk", &linear_chunk);
#endif
#ifdef MB_HAS_ATTENTION
  m.def("window_prep", &window_prep);
  m.def("window_decode", &window_decode);
  m.def("window_attend", &window_attend);
  m.def("window_prefill", &window_prefill);
  m.def("experts_any", &experts_any);
#endif
}
