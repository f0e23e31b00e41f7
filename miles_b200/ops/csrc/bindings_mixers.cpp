// Bindings of the layer-by-layer decoders' kernels: mixers.cu, latent_*.cu, linear_*.cu, window_*.cu, paged_attend.cu, experts_any.cu,
// diff_prep.cu, ssm_*.cu, delta_*.cu.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include "launch.h"

// A serving build (MB_SERVE_SUBSET) has the parts it was asked for (MB_SERVE_…, ops/build.py), any other build all of them.
#if !defined(MB_SERVE_SUBSET)
#define MB_SERVE_LATENT
#define MB_SERVE_LINEAR
#define MB_SERVE_ATTENTION
#define MB_SERVE_PREP
#define MB_SERVE_DIFFERENTIAL
#define MB_SERVE_SSM
#define MB_SERVE_DELTA
#define MB_SERVE_EXPERTS
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
inline long long row_of(const OptTensor& t) { return t.has_value() && t->defined() ? t->stride(0) : 0; }
inline int f32(const at::Tensor& t) { return t.scalar_type() == at::kFloat; }
inline void check(int rc, const char* what) {
  if (rc == 0) return;
  char buf[256];
  snprintf(buf, sizeof(buf), "%s failed with code %d (%s)", what, rc,
           rc > 0 && rc < 1000 ? cudaGetErrorString(static_cast<cudaError_t>(rc)) : "launcher: sizes out of the kernel's range");
  throw std::runtime_error(buf);
}
void bigram_embedding(const at::Tensor& tok, const OptTensor& prev, const at::Tensor& embed, const OptTensor& table, int64_t buckets,
                      int64_t mul_prev, int64_t mul_cur, const OptTensor& positions, const OptTensor& freq, at::Tensor& x, const OptTensor& xb) {
  c10::cuda::CUDAGuard g(embed.device());
  const double* f = freq.has_value() && freq->defined() ? freq->data_ptr<double>() : nullptr;
  TORCH_CHECK(f == nullptr || freq->numel() * 2 >= embed.size(1), "bigram_embedding: a frequency per pair of channels");
  check(mb_bigram_embedding(tok.data_ptr<int>(), iptr(prev), embed.data_ptr(), cptr(table), buckets, mul_prev, mul_cur, iptr(positions), f,
                            x.data_ptr<float>(), mptr(xb), tok.numel(), embed.size(1), f32(embed), cur_stream()),
        "mb_bigram_embedding");
}

void output_norm(at::Tensor& x, const at::Tensor& y, const at::Tensor& nw, const OptTensor& ls, const OptTensor& fw, at::Tensor& xb, double eps,
                 double mult, double gain) {
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(y.is_contiguous() && x.is_contiguous(), "output_norm: contiguous rows");
  check(mb_output_norm(x.data_ptr<float>(), y.data_ptr(), nw.data_ptr(), cptr(ls), mult, cptr(fw), gain, xb.data_ptr(), x.size(0), x.size(1), eps, f32(y),
                       cur_stream()),
        "mb_output_norm");
}

void gemv_output_norm(const at::Tensor& x, const at::Tensor& y, const at::Tensor& nw, const OptTensor& ls, double eps, const at::Tensor& w,
                      at::Tensor& out, at::Tensor& x_out, bool static_w, double mult, const OptTensor& next_w) {
  c10::cuda::CUDAGuard g(x.device());
  check(mb_gemv_output_norm(x.data_ptr<float>(), y.data_ptr(), nw.data_ptr(), cptr(ls), mult, cptr(next_w), eps, w.data_ptr(), out.data_ptr(), out.stride(0),
                            x_out.data_ptr<float>(), x.size(0), w.size(0), x.size(1), static_w, cur_stream()),
        "mb_gemv_output_norm");
}

// rows of `in` [gate, up] and of `out` may be strided; rows (optional): device count of the rows in use
void clamped_glu(const at::Tensor& in, at::Tensor& out, double limit, double alpha, const OptTensor& rows, double shift) {
  c10::cuda::CUDAGuard g(in.device());
  TORCH_CHECK(in.stride(1) == 1 && out.stride(1) == 1 && in.size(1) >= 2 * out.size(1), "clamped_glu: rows of [gate, up]");
  check(mb_clamped_glu(in.data_ptr(), in.stride(0), out.data_ptr(), out.stride(0), out.size(0), out.size(1), limit, alpha, shift, iptr(rows), f32(in),
                       cur_stream()),
        "mb_clamped_glu");
}

void relu_square(at::Tensor& x, const OptTensor& rows) {
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(x.is_contiguous(), "relu_square: contiguous rows");
  check(mb_relu_square(x.data_ptr(), x.size(0), x.size(1), iptr(rows), f32(x), cur_stream()), "mb_relu_square");
}

void part_norm(const at::Tensor& x, const at::Tensor& w, at::Tensor& out, int64_t parts, double eps) {
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(x.stride(1) == 1 && out.is_contiguous() && w.numel() == x.size(1), "part_norm: a weight per channel");
  check(mb_part_norm(x.data_ptr(), x.stride(0), w.data_ptr(), out.data_ptr(), x.size(0), x.size(1), parts, eps, f32(x), cur_stream()), "mb_part_norm");
}

void xielu(const at::Tensor& z, const at::Tensor& act, at::Tensor& out) {
  c10::cuda::CUDAGuard g(z.device());
  TORCH_CHECK(z.is_contiguous() && out.is_contiguous() && act.numel() == 2, "xielu: contiguous values, two numbers");
  check(mb_xielu(z.data_ptr(), act.data_ptr(), out.data_ptr(), z.numel(), f32(z), cur_stream()), "mb_xielu");
}

void gelu_rows(const at::Tensor& z, const at::Tensor& tok, const at::Tensor& table, int64_t col, at::Tensor& out) {
  c10::cuda::CUDAGuard g(z.device());
  TORCH_CHECK(z.stride(1) == 1 && out.is_contiguous() && table.is_contiguous() && col >= 0 && col + z.size(1) <= table.size(1),
              "gelu_rows: columns of the table");
  check(mb_gelu_rows(z.data_ptr(), z.stride(0), tok.data_ptr<int>(), table.data_ptr(), table.size(1), col, out.data_ptr(), z.size(0), z.size(1), f32(z),
                     cur_stream()),
        "mb_gelu_rows");
}

void softcap(at::Tensor& x, double cap, bool exact) {
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(x.is_contiguous(), "softcap: contiguous logits");
  check(mb_softcap(x.data_ptr<float>(), x.numel(), cap, exact, cur_stream()), "mb_softcap");
}

void head_gated_norm(const at::Tensor& o, const at::Tensor& w, const at::Tensor& gate, at::Tensor& out, double eps) {
  c10::cuda::CUDAGuard g(o.device());
  const int64_t V = w.numel();
  TORCH_CHECK(o.is_contiguous() && out.is_contiguous() && gate.stride(1) == 1 && o.size(1) % V == 0, "head_gated_norm: whole heads");
  check(mb_head_gated_norm(o.data_ptr(), w.data_ptr(), gate.data_ptr(), gate.stride(0), out.data_ptr(), o.size(0), o.size(1) / V, V, eps, f32(o),
                           cur_stream()),
        "mb_head_gated_norm");
}

// every addend may have a scale (s1 of y1; s2 of y2 or of the experts' rows)
void sum_norm(const at::Tensor& x, const OptTensor& to, const OptTensor& y1, const OptTensor& s1, const OptTensor& y2, const OptTensor& s2,
              const OptTensor& rows, const OptTensor& weights, const OptTensor& dst, const OptTensor& extra, const OptTensor& nw, const OptTensor& h,
              const OptTensor& nw2, const OptTensor& h2, double eps, double shift, double gain, double mult) {
  c10::cuda::CUDAGuard g(x.device());
  MbSumNorm p{};
  p.x = x.data_ptr<float>();
  p.to = fmut(to);
  p.y1 = cptr(y1);
  p.y2 = cptr(y2);
  p.s1 = cptr(s1);
  p.s2 = cptr(s2);
  p.rows = cptr(rows);
  p.weights = fptr(weights);
  p.dst = iptr(dst);
  p.extra = fptr(extra);
  p.nw = cptr(nw);
  p.h = mptr(h);
  p.nw2 = cptr(nw2);
  p.h2 = mptr(h2);
  p.T = x.size(0);
  p.D = x.size(1);
  p.k = p.weights != nullptr ? weights->size(1) : 0;
  p.eps = eps;
  p.shift = shift;
  p.gain = gain;
  p.mult = mult;
  for (const OptTensor* t : {&y1, &y2, &rows, &nw, &nw2, &s1, &s2})
    TORCH_CHECK(!t->has_value() || !(*t)->defined() || (*t)->is_contiguous(), "sum_norm: contiguous rows");
  TORCH_CHECK(p.s2 == nullptr || p.y2 == nullptr || p.rows == nullptr, "sum_norm: one addend per scale");
  int is32 = 0;
  for (const OptTensor* t : {&nw, &y1, &y2, &rows, &h})
    if (t->has_value() && (*t)->defined()) is32 = f32(**t);
  check(mb_sum_norm(p, is32, cur_stream()), "mb_sum_norm");
}

// x32 (with y1·s1, y2·s2, extra, norm_w) or plain rows x; W [N, K] → y, W2 [N2, K] → y2out (float or bf16; its rows by norm_w2 if given)
void gemv_sum_norm(const OptTensor& x32, const OptTensor& y1, const OptTensor& s1, const OptTensor& y2, const OptTensor& s2, const OptTensor& extra,
                   const OptTensor& x, const OptTensor& norm_w, const OptTensor& norm_w2, double eps, double shift, const at::Tensor& W, at::Tensor& y,
                   const OptTensor& W2, const OptTensor& bias2, const OptTensor& y2out, const OptTensor& x_out, const OptTensor& xn_out, bool static_w,
                   double mult, const OptTensor& x2) {
  c10::cuda::CUDAGuard g(W.device());
  const bool two = W2.has_value() && W2->defined();
  MbGemvSum a{};
  a.x32 = fptr(x32);
  a.y1 = cptr(y1);
  a.s1 = cptr(s1);
  a.y2 = cptr(y2);
  a.s2 = cptr(s2);
  a.extra = fptr(extra);
  a.x = cptr(x);
  a.x2 = cptr(x2);
  a.ldx = a.x != nullptr && x->size(0) > 1 ? row_of(x) : W.size(1);
  TORCH_CHECK(a.x2 == nullptr || x->size(0) == 1 || row_of(x2) == a.ldx, "gemv_sum_norm: both rows out of one matrix");
  a.norm_w = cptr(norm_w);
  a.norm_w2 = cptr(norm_w2);
  a.eps = eps;
  a.shift = shift;
  a.mult = mult;
  a.W = W.data_ptr();
  a.y = y.data_ptr();
  a.ldy = y.stride(0);
  a.W2 = cptr(W2);
  a.bias2 = cptr(bias2);
  if (two) {
    a.out2 = mptr(y2out);
    a.ld2 = y2out->stride(0);
    a.out2_fp32 = f32(*y2out);
    a.N2 = W2->size(0);
  }
  a.x_out = fmut(x_out);
  a.xn_out = mptr(xn_out);
  a.M = y.size(0);
  a.N = W.size(0);
  a.K = W.size(1);
  a.static_w = static_w;
  check(mb_gemv_sum_norm(a, cur_stream()), "mb_gemv_sum_norm");
}

void gated_norm(const at::Tensor& o, const at::Tensor& w, const at::Tensor& gate, at::Tensor& out, double eps) {
  c10::cuda::CUDAGuard g(o.device());
  check(mb_gated_norm(o.data_ptr(), w.data_ptr(), gate.data_ptr(), gate.stride(0), out.data_ptr(), o.size(0), o.size(1), eps, f32(o), cur_stream()),
        "mb_gated_norm");
}

#ifdef MB_SERVE_LATENT
inline MbLatent layout(const std::vector<int64_t>& v) {
  TORCH_CHECK(v.size() == 7, "latent layout has 7 sizes");
  return MbLatent{static_cast<int>(v[0]), static_cast<int>(v[1]), static_cast<int>(v[2]), static_cast<int>(v[3]),
                  static_cast<int>(v[4]), static_cast<int>(v[5]), static_cast<int>(v[6])};
}

void latent_prep(const at::Tensor& q, const at::Tensor& kv, const at::Tensor& positions, const at::Tensor& slots, const at::Tensor& freq, double magnitude,
                 const OptTensor& kv_norm, double eps, at::Tensor& cache, const OptTensor& q_abs, const OptTensor& q_full, int64_t t_long,
                 int64_t q_nope, int64_t q_width, const std::vector<int64_t>& lay) {
  c10::cuda::CUDAGuard g(q.device());
  TORCH_CHECK(q.stride(1) == 1 && (kv.size(1) == 0 || kv.stride(1) == 1), "latent_prep: rows");
  check(mb_latent_prep(q.data_ptr(), q.stride(0), kv.data_ptr(), kv.stride(0), positions.data_ptr<int>(), lptr(slots), freq.data_ptr<double>(), magnitude,
                       cptr(kv_norm), eps, cache.data_ptr(), mptr(q_abs), mptr(q_full), q.size(0), t_long, q_nope, q_width, layout(lay), f32(q),
                       cur_stream()),
        "mb_latent_prep");
}

// x [T, H, K] (any strides of T and H), w [H, N, K] (w_nk) or [H, K, N], y [T, H, N] (any strides of T and H)
void head_linear(const at::Tensor& x, const at::Tensor& w, bool w_nk, at::Tensor& y, const OptTensor& gate) {
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(x.stride(2) == 1 && y.stride(2) == 1 && w.is_contiguous(), "head_linear: innermost dimension must be contiguous");
  check(mb_head_linear(x.data_ptr(), x.stride(0), x.stride(1), w.data_ptr(), w_nk, y.data_ptr(), y.stride(0), y.stride(1), x.size(0), x.size(1),
                       y.size(2), x.size(2), cptr(gate), row_of(gate), f32(x), cur_stream()),
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

void head_linear_mma(const at::Tensor& x, const at::Tensor& w, bool w_nk, at::Tensor& y, const OptTensor& gate) {
  c10::cuda::CUDAGuard g(x.device());
  TORCH_CHECK(x.stride(2) == 1 && y.stride(2) == 1 && w.is_contiguous(), "head_linear_mma: innermost dimension must be contiguous");
  check(mb_head_linear_mma(x.data_ptr(), x.stride(0), x.stride(1), w.data_ptr(), w_nk, y.data_ptr(), y.stride(0), y.stride(1), x.size(0),
                           x.size(1), y.size(2), x.size(2), cptr(gate), row_of(gate), cur_stream()),
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
                    at::Tensor& err, const OptTensor& gate) {
  c10::cuda::CUDAGuard g(q.device());
  check(mb_latent_prefill(q.data_ptr(), kv.data_ptr(), lat.data_ptr(), o.data_ptr(), cptr(sink), cptr(gate), row_of(gate), cu_q.data_ptr<int>(), cu_k.data_ptr<int>(), n_seq,
                          max_q, q.size(0), lat.size(0), scale, window, layout(lay), err.data_ptr<int>(), cur_stream()),
        "mb_latent_prefill");
}

#endif  // MB_SERVE_LATENT

#ifdef MB_SERVE_LINEAR
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
#endif  // MB_SERVE_LINEAR

// {logits, weights, index, glu_in, glu_out, correction (each or None)}, {limit, alpha, up shift, weights' scale}, {grouped, groups, keep}
[[maybe_unused]] inline MbAside aside(const std::vector<OptTensor>& t, const std::vector<double>& f, const std::vector<int64_t>& n) {
  TORCH_CHECK(t.size() == 6 && f.size() == 4 && n.size() == 3, "an aside has 6 tensors, 4 numbers and 3 counts");
  MbAside a{};
  if (t[0].has_value() && t[0]->defined()) {
    a.logits = t[0]->data_ptr<float>();
    a.weights = fmut(t[1]);
    a.index = t[2]->data_ptr<int>();
    a.experts = t[0]->size(1);
    a.top = t[2]->size(1);
    TORCH_CHECK(t[0]->is_contiguous(), "an aside's logits are contiguous");
  }
  if (t[3].has_value() && t[3]->defined()) {
    a.glu_in = t[3]->data_ptr();
    a.glu_out = mptr(t[4]);
    a.glu_ld_in = t[3]->stride(0);
    a.glu_ld_out = t[4]->stride(0);
    a.ff = t[4]->size(1);
  }
  a.correction = cptr(t[5]);
  a.limit = f[0];
  a.alpha = f[1];
  a.shift = f[2];
  a.scale = f[3];
  a.grouped = n[0];
  a.groups = n[1];
  a.keep = n[2];
  return a;
}

// (weight of the second map, gate rows, gain, eps), or nothing
[[maybe_unused]] inline MbDiff difference(const OptTensor& lam, const OptTensor& gate, double gain, double eps) {
  MbDiff d{};
  d.lam = fptr(lam);
  if (d.lam == nullptr) return d;
  TORCH_CHECK(gate.has_value() && gate->stride(1) == 1, "differential attention has gates, one per head");
  d.gate = gate->data_ptr();
  d.gate_ld = gate->stride(0);
  d.gain = gain;
  d.eps = eps;
  return d;
}

[[maybe_unused]] inline MbWindow window(const std::vector<int64_t>& v) {
  TORCH_CHECK(v.size() == 8 || v.size() == 9, "a windowed attention layout has 8 sizes, and a chunk size if there are chunks");
  return MbWindow{static_cast<int>(v[0]), static_cast<int>(v[1]), static_cast<int>(v[2]), static_cast<int>(v[3]), static_cast<int>(v[4]),
                  static_cast<int>(v[5]), static_cast<int>(v[6]), static_cast<int>(v[7]), v.size() == 9 ? static_cast<int>(v[8]) : 0};
}

#ifdef MB_SERVE_PREP
// kc, vc None: another layer's keys and values
void window_prep(const at::Tensor& proj, const at::Tensor& positions, const at::Tensor& slots, const at::Tensor& freq, double magnitude,
                 const OptTensor& q_norm, const OptTensor& k_norm, double eps, const OptTensor& kc, const OptTensor& vc, at::Tensor& q,
                 const std::vector<int64_t>& lay, const std::vector<OptTensor>& at, const std::vector<double>& af, const std::vector<int64_t>& an,
                 bool v_norm) {
  c10::cuda::CUDAGuard g(proj.device());
  check(mb_window_prep(proj.data_ptr(), proj.stride(0), positions.data_ptr<int>(), lptr(slots), freq.data_ptr<double>(), magnitude, cptr(q_norm),
                       cptr(k_norm), v_norm, eps, mptr(kc), mptr(vc), q.data_ptr(), proj.size(0), window(lay), aside(at, af, an), f32(proj),
                       cur_stream()),
        "mb_window_prep");
}
#endif

#ifdef MB_SERVE_ATTENTION
// r1, r2: distance bias per head; gate: rows of heads·vdim
inline MbScores scores(const OptTensor& r1, const OptTensor& r2, const OptTensor& gate, const at::Tensor& like, int heads) {
  MbScores x{};
  x.r1 = cptr(r1);
  x.r2 = cptr(r2);
  TORCH_CHECK((x.r1 == nullptr) == (x.r2 == nullptr) && (x.r1 == nullptr || (r1->numel() == heads && r2->numel() == heads && r1->scalar_type() == like.scalar_type() &&
                                                                             r2->scalar_type() == like.scalar_type())), "a distance bias has two numbers per head");
  x.gate = cptr(gate);
  x.gate_ld = row_of(gate);
  TORCH_CHECK(x.gate == nullptr || (gate->stride(1) == 1 && gate->scalar_type() == like.scalar_type()), "gates are rows of the outputs' type");
  return x;
}

void window_decode(const at::Tensor& q, const at::Tensor& kc, const at::Tensor& vc, const at::Tensor& block_table, const OptTensor& token_seq,
                   const at::Tensor& positions, const at::Tensor& slots, const OptTensor& sink, at::Tensor& out, double scale, int64_t splits,
                   const std::vector<int64_t>& lay, const OptTensor& lam, const OptTensor& gate, double gain, double eps, const OptTensor& r1,
                   const OptTensor& r2, const OptTensor& out_gate) {
  c10::cuda::CUDAGuard g(q.device());
  check(mb_window_decode(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), block_table.data_ptr<int>(), block_table.size(1), kc.size(1), iptr(token_seq),
                         positions.data_ptr<int>(), lptr(slots), cptr(sink), out.data_ptr(), out.stride(0), q.size(0), scale, splits, window(lay),
                         difference(lam, gate, gain, eps), scores(r1, r2, out_gate, q, lay[0]), cur_stream()),
        "mb_window_decode");
}

void window_attend(const at::Tensor& q, const at::Tensor& kc, const at::Tensor& vc, const at::Tensor& block_table, const OptTensor& token_seq,
                   const at::Tensor& positions, const at::Tensor& slots, const OptTensor& sink, at::Tensor& out, double scale,
                   const std::vector<int64_t>& lay, const OptTensor& r1, const OptTensor& r2, const OptTensor& out_gate) {
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
  a.chunk = L.chunk;
  a.scale = scale;
  check(mb_paged_attend(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), block_table.data_ptr<int>(), block_table.size(1), kc.size(1), iptr(token_seq),
                        positions.data_ptr<int>(), lptr(slots), cptr(sink), out.data_ptr(), q.size(0), a, scores(r1, r2, out_gate, q, L.heads), f32(q), f32(out), cur_stream()),
        "mb_paged_attend");
}

void window_prefill(const at::Tensor& q, const at::Tensor& kc, const at::Tensor& vc, at::Tensor& out, const OptTensor& sink, const at::Tensor& cu_q,
                    const at::Tensor& positions, const at::Tensor& block_table, int64_t n_seq, int64_t max_q, int64_t t_long, double scale,
                    const std::vector<int64_t>& lay, at::Tensor& err, const OptTensor& lam, const OptTensor& gate, double gain, double eps,
                    const OptTensor& r1, const OptTensor& r2, const OptTensor& out_gate) {
  c10::cuda::CUDAGuard g(q.device());
  check(mb_window_prefill(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), out.data_ptr(), out.stride(0), cptr(sink), cu_q.data_ptr<int>(),
                          positions.data_ptr<int>(), block_table.data_ptr<int>(), block_table.size(1), kc.size(1), kc.size(0), n_seq, max_q, t_long,
                          scale, window(lay), difference(lam, gate, gain, eps), scores(r1, r2, out_gate, q, lay[0]), err.data_ptr<int>(), cur_stream()),
        "mb_window_prefill");
}

#endif  // MB_SERVE_ATTENTION

#ifdef MB_SERVE_EXPERTS
void experts_any(const at::Tensor& x, const at::Tensor& w13, const at::Tensor& w2, const at::Tensor& index, const at::Tensor& weights, at::Tensor& act,
                 at::Tensor& out, double limit, double alpha, double shift) {
  c10::cuda::CUDAGuard g(x.device());
  mb_count_launch(1);
  check(mb_experts_any(x.data_ptr(), w13.data_ptr(), w2.data_ptr(), index.data_ptr<int>(), weights.data_ptr<float>(), act.data_ptr(), out.data_ptr(),
                       x.size(0), index.size(1), w13.size(0), x.size(1), w2.size(2), limit, alpha, shift, f32(x), cur_stream()),
        "mb_experts_any");
}
#endif  // MB_SERVE_EXPERTS

#ifdef MB_SERVE_DIFFERENTIAL
// sizes: heads, key heads (0: another layer's keys and values), one map's size, value size, elements per prepared query row
void diff_prep(const at::Tensor& proj, const at::Tensor& positions, const at::Tensor& slots, const at::Tensor& q_norm, const OptTensor& k_norm,
               const at::Tensor& lvec, at::Tensor& lam, const OptTensor& kc, const OptTensor& vc, at::Tensor& q, const std::vector<int64_t>& sizes,
               double eps, double temp_coef, double temp_every, double diff, const std::vector<OptTensor>& at, const std::vector<double>& af,
               const std::vector<int64_t>& an) {
  c10::cuda::CUDAGuard g(proj.device());
  TORCH_CHECK(sizes.size() == 5 && lvec.is_contiguous(), "diff_prep: 5 sizes, stacked vectors");
  const MbDiffPrep L{static_cast<int>(sizes[0]), static_cast<int>(sizes[1]), static_cast<int>(sizes[2]), static_cast<int>(sizes[3]),
                     static_cast<int>(sizes[4]), static_cast<float>(eps), static_cast<float>(temp_coef), temp_every, static_cast<float>(diff)};
  check(mb_diff_prep(proj.data_ptr(), proj.stride(0), positions.data_ptr<int>(), lptr(slots), q_norm.data_ptr(), cptr(k_norm), lvec.data_ptr(),
                     lam.data_ptr<float>(), mptr(kc), mptr(vc), q.data_ptr(), proj.size(0), L, aside(at, af, an), f32(proj), cur_stream()),
        "mb_diff_prep");
}

void diff_combine(const at::Tensor& a, at::Tensor& out, int64_t heads, int64_t vdim, const OptTensor& lam, const OptTensor& gate, double gain, double eps) {
  c10::cuda::CUDAGuard g(a.device());
  check(mb_diff_combine(a.data_ptr<float>(), out.data_ptr(), out.stride(0), out.size(0), heads, vdim, difference(lam, gate, gain, eps), f32(out),
                        cur_stream()),
        "mb_diff_combine");
}

#endif  // MB_SERVE_DIFFERENTIAL

#ifdef MB_SERVE_SSM
// sizes: heads, value size, state size, groups, taps; t: conv weight, conv bias, dt_bias, A_log, D, state, ring (or None), slots, positions
inline MbSsm ssm(const std::vector<int64_t>& sizes, const std::vector<OptTensor>& t) {
  TORCH_CHECK(sizes.size() == 5 && t.size() == 9, "a state-space mixer has 5 sizes and 9 tensors");
  MbSsm m{};
  m.H = sizes[0];
  m.V = sizes[1];
  m.N = sizes[2];
  m.G = sizes[3];
  m.taps = sizes[4];
  m.conv_w = cptr(t[0]);
  m.conv_b = cptr(t[1]);
  m.dt_bias = cptr(t[2]);
  m.A_log = cptr(t[3]);
  m.D = cptr(t[4]);
  m.state = fmut(t[5]);
  m.ring = fmut(t[6]);
  m.slots = iptr(t[7]);
  m.positions = iptr(t[8]);
  return m;
}

void ssm_conv(const at::Tensor& proj, const std::vector<int64_t>& sizes, const std::vector<OptTensor>& t, const OptTensor& tiles, const OptTensor& cu_q,
              at::Tensor& xbc, at::Tensor& dt, at::Tensor& la, const std::vector<OptTensor>& at, const std::vector<double>& af,
              const std::vector<int64_t>& an) {
  c10::cuda::CUDAGuard g(proj.device());
  const bool given = tiles.has_value() && tiles->defined();
  check(mb_ssm_conv(proj.data_ptr(), proj.stride(0), ssm(sizes, t), iptr(tiles), iptr(cu_q), given ? tiles->size(0) : proj.size(0), xbc.data_ptr(),
                    dt.data_ptr<float>(), la.data_ptr<float>(), proj.size(0), aside(at, af, an), f32(proj), cur_stream()),
        "mb_ssm_conv");
}

void ssm_step(const at::Tensor& proj, const std::vector<int64_t>& sizes, const std::vector<OptTensor>& t, at::Tensor& out,
              const std::vector<OptTensor>& at, const std::vector<double>& af, const std::vector<int64_t>& an) {
  c10::cuda::CUDAGuard g(proj.device());
  check(mb_ssm_step(proj.data_ptr(), proj.stride(0), ssm(sizes, t), out.data_ptr(), proj.size(0), aside(at, af, an), f32(proj), cur_stream()),
        "mb_ssm_step");
}

void ssm_seq(const at::Tensor& proj, const at::Tensor& xbc, const at::Tensor& dt, const at::Tensor& la, const std::vector<int64_t>& sizes,
             const std::vector<OptTensor>& t, const OptTensor& cu_q, at::Tensor& out) {
  c10::cuda::CUDAGuard g(proj.device());
  check(mb_ssm_seq(proj.data_ptr(), proj.stride(0), xbc.data_ptr(), dt.data_ptr<float>(), la.data_ptr<float>(), ssm(sizes, t), iptr(cu_q),
                   out.data_ptr(), t[7]->numel(), f32(proj), cur_stream()),
        "mb_ssm_seq");
}

void ssm_chunk(const at::Tensor& proj, const at::Tensor& xbc, const at::Tensor& dt, const at::Tensor& la, const std::vector<int64_t>& sizes,
               const std::vector<OptTensor>& t, const at::Tensor& segs, const at::Tensor& seq_segs, const OptTensor& seg_state, const OptTensor& seg_decay,
               at::Tensor& out) {
  c10::cuda::CUDAGuard g(proj.device());
  if (fptr(seg_state) != nullptr) mb_count_launch(2);
  check(mb_ssm_chunk(proj.data_ptr(), proj.stride(0), xbc.data_ptr(), dt.data_ptr<float>(), la.data_ptr<float>(), ssm(sizes, t), segs.data_ptr<int>(),
                     seq_segs.data_ptr<int>(), fmut(seg_state), fmut(seg_decay), out.data_ptr(), seq_segs.numel() - 1, segs.size(0), cur_stream()),
        "mb_ssm_chunk");
}
#endif  // MB_SERVE_SSM

#ifdef MB_SERVE_DELTA
// sizes: heads, query/key heads, key size, value size, taps, column of β; t: conv weight, A_log, dt_bias, state, ring (or None), slots, positions,
// raw decays
inline MbDelta delta(const std::vector<int64_t>& sizes, const std::vector<OptTensor>& t) {
  TORCH_CHECK(sizes.size() == 6 && t.size() == 8, "a delta-rule mixer has 6 sizes and 8 tensors");
  MbDelta m{};
  m.H = sizes[0];
  m.G = sizes[1];
  m.K = sizes[2];
  m.V = sizes[3];
  m.taps = sizes[4];
  m.beta_at = sizes[5];
  m.conv_w = cptr(t[0]);
  m.A_log = cptr(t[1]);
  m.dt_bias = cptr(t[2]);
  m.state = fmut(t[3]);
  m.ring = fmut(t[4]);
  m.slots = iptr(t[5]);
  m.positions = iptr(t[6]);
  m.raw = cptr(t[7]);
  m.raw_ld = row_of(t[7]);
  return m;
}

void delta_conv(const at::Tensor& proj, const std::vector<int64_t>& sizes, const std::vector<OptTensor>& t, const OptTensor& tiles, const OptTensor& cu_q,
                at::Tensor& act) {
  c10::cuda::CUDAGuard g(proj.device());
  const bool given = tiles.has_value() && tiles->defined();
  check(mb_delta_conv(proj.data_ptr(), proj.stride(0), delta(sizes, t), iptr(tiles), iptr(cu_q), given ? tiles->size(0) : proj.size(0), act.data_ptr(),
                      f32(proj), cur_stream()),
        "mb_delta_conv");
}

void delta_seq(const at::Tensor& proj, const at::Tensor& act, const std::vector<int64_t>& sizes, const std::vector<OptTensor>& t, const OptTensor& cu_q,
               at::Tensor& out) {
  c10::cuda::CUDAGuard g(proj.device());
  check(mb_delta_seq(proj.data_ptr(), proj.stride(0), act.data_ptr(), delta(sizes, t), iptr(cu_q), out.data_ptr(), t[5]->numel(), f32(proj), cur_stream()),
        "mb_delta_seq");
}

void delta_chunk(const at::Tensor& proj, const at::Tensor& act, const std::vector<int64_t>& sizes, const std::vector<OptTensor>& t, const at::Tensor& chunks,
                 const at::Tensor& parts, at::Tensor& scratch, int64_t warps, at::Tensor& out, at::Tensor& err) {
  c10::cuda::CUDAGuard g(proj.device());
  const MbDelta m = delta(sizes, t);
  TORCH_CHECK(scratch.nbytes() >= static_cast<size_t>(mb_delta_chunk_bytes(m.K, m.V)) * chunks.size(0) * m.H, "delta_chunk: scratch too small");
  mb_count_launch(1);
  check(mb_delta_chunk(proj.data_ptr(), proj.stride(0), act.data_ptr(), m, chunks.data_ptr<int>(), parts.data_ptr<int>(), scratch.data_ptr(),
                       out.data_ptr(), proj.size(0), chunks.size(0), parts.size(0), warps, err.data_ptr<int>(), cur_stream()),
        "mb_delta_chunk");
}

void delta_step(const at::Tensor& proj, const std::vector<int64_t>& sizes, const std::vector<OptTensor>& t, const at::Tensor& norm_w, const at::Tensor& gate,
                double eps, at::Tensor& out) {
  c10::cuda::CUDAGuard g(proj.device());
  check(mb_delta_step(proj.data_ptr(), proj.stride(0), delta(sizes, t), norm_w.data_ptr(), gate.data_ptr(), gate.stride(0), eps, out.data_ptr(),
                      proj.size(0), f32(proj), cur_stream()),
        "mb_delta_step");
}
#endif  // MB_SERVE_DELTA

}  // namespace

void register_mixers(pybind11::module& m) {
  m.def("bigram_embedding", &bigram_embedding);
  using pybind11::arg;
  m.def("output_norm", &output_norm, arg("x"), arg("y"), arg("nw"), arg("ls"), arg("fw"), arg("xb"), arg("eps"), arg("mult") = 1.0, arg("gain") = 1.0);
  m.def("gemv_output_norm", &gemv_output_norm, arg("x"), arg("y"), arg("nw"), arg("ls"), arg("eps"), arg("w"), arg("out"), arg("x_out"), arg("static_w"),
        arg("mult") = 1.0, arg("next_w") = pybind11::none());
  m.def("xielu", &xielu);
  m.def("gelu_rows", &gelu_rows);
  m.def("softcap", &softcap);
  m.def("head_gated_norm", &head_gated_norm);
  m.def("clamped_glu", &clamped_glu, pybind11::arg("in"), pybind11::arg("out"), pybind11::arg("limit"), pybind11::arg("alpha"),
        pybind11::arg("rows") = pybind11::none(), pybind11::arg("shift") = 1.0);
  m.def("sum_norm", &sum_norm, arg("x"), arg("to"), arg("y1"), arg("s1"), arg("y2"), arg("s2"), arg("rows"), arg("weights"), arg("dst"), arg("extra"),
        arg("nw"), arg("h"), arg("nw2"), arg("h2"), arg("eps"), arg("shift"), arg("gain"), arg("mult") = 1.0);
  m.def("gemv_sum_norm", &gemv_sum_norm, arg("x32"), arg("y1"), arg("s1"), arg("y2"), arg("s2"), arg("extra"), arg("x"), arg("norm_w"), arg("norm_w2"),
        arg("eps"), arg("shift"), arg("W"), arg("y"), arg("W2"), arg("bias2"), arg("y2out"), arg("x_out"), arg("xn_out"), arg("static_w"), arg("mult") = 1.0,
        arg("x2") = pybind11::none());
  m.def("gated_norm", &gated_norm);
  m.def("relu_square", &relu_square, pybind11::arg("x"), pybind11::arg("rows") = pybind11::none());
  m.def("part_norm", &part_norm);
#ifdef MB_SERVE_LATENT
  m.def("latent_prep", &latent_prep);
  m.def("head_linear", &head_linear, arg("x"), arg("w"), arg("w_nk"), arg("y"), arg("gate") = pybind11::none());
  m.def("latent_attend", &latent_attend);
  m.def("latent_gather", &latent_gather);
  m.def("head_linear_mma", &head_linear_mma, arg("x"), arg("w"), arg("w_nk"), arg("y"), arg("gate") = pybind11::none());
  m.def("latent_decode", &latent_decode);
  m.def("latent_prefill", &latent_prefill, arg("q"), arg("kv"), arg("lat"), arg("o"), arg("sink"), arg("cu_q"), arg("cu_k"), arg("n_seq"), arg("max_q"),
        arg("scale"), arg("window"), arg("lay"), arg("err"), arg("gate") = pybind11::none());
#endif
#ifdef MB_SERVE_LINEAR
  m.def("linear_state", &linear_state);
  m.def("linear_chunk", &linear_chunk);
#endif
#ifdef MB_SERVE_PREP
  m.def("window_prep", &window_prep, arg("proj"), arg("positions"), arg("slots"), arg("freq"), arg("magnitude"), arg("q_norm"), arg("k_norm"), arg("eps"),
        arg("kc"), arg("vc"), arg("q"), arg("lay"), arg("at"), arg("af"), arg("an"), arg("v_norm") = false);
#endif
#ifdef MB_SERVE_DELTA
  m.def("delta_conv", &delta_conv);
  m.def("delta_seq", &delta_seq);
  m.def("delta_step", &delta_step);
  m.def("delta_step_ok", &mb_delta_step_ok);
  m.def("delta_chunk", &delta_chunk);
  m.def("delta_chunk_bytes", &mb_delta_chunk_bytes);
#endif
#ifdef MB_SERVE_DIFFERENTIAL
  m.def("diff_prep", &diff_prep);
  m.def("diff_combine", &diff_combine);
#endif
#ifdef MB_SERVE_SSM
  m.def("ssm_conv", &ssm_conv);
  m.def("ssm_step", &ssm_step);
  m.def("ssm_seq", &ssm_seq);
  m.def("ssm_chunk", &ssm_chunk);
  m.def("ssm_heads_per_cta", &mb_ssm_heads_per_cta);
#endif
#ifdef MB_SERVE_ATTENTION
  m.def("window_decode", &window_decode, pybind11::arg("q"), pybind11::arg("kc"), pybind11::arg("vc"), pybind11::arg("block_table"), pybind11::arg("token_seq"), pybind11::arg("positions"),
        pybind11::arg("slots"), pybind11::arg("sink"), pybind11::arg("out"), pybind11::arg("scale"), pybind11::arg("splits"), pybind11::arg("lay"),
        pybind11::arg("lam") = pybind11::none(), pybind11::arg("gate") = pybind11::none(), pybind11::arg("gain") = 0.0, pybind11::arg("eps") = 0.0,
        arg("r1") = pybind11::none(), arg("r2") = pybind11::none(), arg("out_gate") = pybind11::none());
  m.def("window_attend", &window_attend, arg("q"), arg("kc"), arg("vc"), arg("block_table"), arg("token_seq"), arg("positions"), arg("slots"), arg("sink"),
        arg("out"), arg("scale"), arg("lay"), arg("r1") = pybind11::none(), arg("r2") = pybind11::none(), arg("out_gate") = pybind11::none());
  m.def("window_prefill", &window_prefill, pybind11::arg("q"), pybind11::arg("kc"), pybind11::arg("vc"), pybind11::arg("out"), pybind11::arg("sink"), pybind11::arg("cu_q"), pybind11::arg("positions"),
        pybind11::arg("block_table"), pybind11::arg("n_seq"), pybind11::arg("max_q"), pybind11::arg("t_long"), pybind11::arg("scale"), pybind11::arg("lay"), pybind11::arg("err"),
        pybind11::arg("lam") = pybind11::none(), pybind11::arg("gate") = pybind11::none(), pybind11::arg("gain") = 0.0, pybind11::arg("eps") = 0.0,
        arg("r1") = pybind11::none(), arg("r2") = pybind11::none(), arg("out_gate") = pybind11::none());
#endif
#ifdef MB_SERVE_EXPERTS
  m.def("experts_any", &experts_any, pybind11::arg("x"), pybind11::arg("w13"), pybind11::arg("w2"), pybind11::arg("index"), pybind11::arg("weights"),
        pybind11::arg("act"), pybind11::arg("out"), pybind11::arg("limit"), pybind11::arg("alpha"), pybind11::arg("shift") = 1.0);
#endif
}
