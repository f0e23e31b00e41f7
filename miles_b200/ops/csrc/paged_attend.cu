// Attention of single tokens over a paged cache of keys and values, any sizes (bf16 or float): the form that runs where no
// tensor-core kernel fits, and every 32-bit run.
//
// A token at position p sees the keys less than `window` back (0: all) and the first `keep` ones, or those of its own chunk.  Query
// head h uses key head h / group.  The softmax has an optional sink per head; scores may lose a distance bias, outputs pass a gate (MbScores).
#include "mixers.cuh"

namespace mb {
namespace mx {

// grid (heads, tokens), 128 threads: each warp takes every fourth key with its own running softmax; RL · 32 ≥ dv.
template <typename T, typename O, int RL>
__global__ void __launch_bounds__(128) paged_attend_kernel(const T* __restrict__ q, const T* __restrict__ kc, const T* __restrict__ vc,
                                                           const int* __restrict__ block_table, int max_blocks, int block_size,
                                                           const int* __restrict__ token_seq, const int* __restrict__ positions,
                                                           const long long* __restrict__ slots, const T* __restrict__ sink,
                                                           O* __restrict__ out, MbAttend A, MbScores x) {
  extern __shared__ float sm[];
  float* sq = sm;                        // [dk]
  float* so = sq + A.dk;                 // [4][dv]
  __shared__ float s_m[4], s_l[4];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.y;
  const int h = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  O* o = out + t * A.o_row + static_cast<long long>(h) * A.dv;
  if (slots[t] < 0) {                    // padding row of a decode batch
    for (int i = threadIdx.x; i < A.dv; i += 128) o[i] = from_f<O>(0.f);
    return;
  }
  const int pos = positions[t];
  const int lo = A.window > 0 ? max(0, pos - A.window + 1) : A.chunk > 0 ? pos - pos % A.chunk : 0;
  const float r1 = x.r1 != nullptr ? to_f(reinterpret_cast<const T*>(x.r1)[h]) : 0.f, r2 = x.r1 != nullptr ? to_f(reinterpret_cast<const T*>(x.r2)[h]) : 0.f;
  const int kept = min(A.keep, lo);      // keys before the window that stay visible
  const int* bt = block_table + static_cast<long long>(token_seq != nullptr ? token_seq[t] : t) * max_blocks;
  const long long k_at = static_cast<long long>(h / A.group) * A.k_head, v_at = static_cast<long long>(h / A.group) * A.v_head;
  for (int i = threadIdx.x; i < A.dk; i += 128) sq[i] = to_f(q[t * A.q_row + h * A.q_head + i]);
  __syncthreads();
  float m = -INFINITY, l = 0.f, acc[RL];
#pragma unroll
  for (int i = 0; i < RL; ++i) acc[i] = 0.f;
  for (int i = warp; i < kept + pos + 1 - lo; i += 4) {
    const int key = i < kept ? i : lo + i - kept;
    const long long slot = static_cast<long long>(bt[key / block_size]) * block_size + key % block_size;
    const T* kr = kc + slot * A.k_row + k_at;
    const T* vr = vc + slot * A.v_row + v_at;
    float v[RL], s = 0.f;
#pragma unroll
    for (int j = 0; j < RL; ++j) {
      const int c = lane + 32 * j;
      v[j] = c < A.dv ? to_f(vr[c]) : 0.f;
    }
    for (int c = lane; c < A.dk; c += 32) s = fmaf(to_f(kr[c]), sq[c], s);
    s = warp_sum(s) * A.scale;
    if (x.r1 != nullptr) {
      if constexpr (is_exact<T>::value) s -= r1 * static_cast<float>(log1p(static_cast<double>(r2) * (pos - key)));
      else s -= r1 * __logf(fmaf(r2, static_cast<float>(pos - key), 1.f));
    }
    const float mn = fmaxf(m, s);
    const float a = exp_t<T>(m - mn), p = exp_t<T>(s - mn);
    m = mn;
    l = fmaf(l, a, p);
#pragma unroll
    for (int j = 0; j < RL; ++j) acc[j] = fmaf(acc[j], a, p * v[j]);
  }
#pragma unroll
  for (int i = 0; i < RL; ++i) {
    const int c = lane + 32 * i;
    if (c < A.dv) so[warp * A.dv + c] = acc[i];
  }
  if (lane == 0) { s_m[warp] = m; s_l[warp] = l; }
  __syncthreads();
  float mm = sink != nullptr ? to_f(sink[h]) : -INFINITY;
#pragma unroll
  for (int w = 0; w < 4; ++w) mm = fmaxf(mm, s_m[w]);
  float f[4], den = sink != nullptr ? exp_t<T>(to_f(sink[h]) - mm) : 0.f;
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    f[w] = s_m[w] == -INFINITY ? 0.f : exp_t<T>(s_m[w] - mm);
    den = fmaf(s_l[w], f[w], den);
  }
  for (int i = threadIdx.x; i < A.dv; i += 128) {
    float r = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) r = fmaf(so[w * A.dv + i], f[w], r);
    r = __fdiv_rn(r, den);
    if (x.gate != nullptr) r *= sigmoid_t<T>(to_f(reinterpret_cast<const T*>(x.gate)[t * x.gate_ld + h * A.dv + i]));
    o[i] = from_f<O>(r);
  }
}

template <typename T, typename O, int RL>
static int attend_rl(const T* q, const T* kc, const T* vc, const int* bt, int mb_, int bs, const int* seq, const int* pos, const long long* slots,
                     const T* sink, O* out, int n, MbAttend A, MbScores x, cudaStream_t s) {
  const size_t bytes = (A.dk + 4 * A.dv) * sizeof(float);
  if (bytes > 48 * 1024) return -3;
  if (seq == nullptr && n > 65535) return -3;      // a decode batch (token = row) never gets this large
  for (int t0 = 0; t0 < n; t0 += 65535) {
    MbScores xt = x;
    if (x.gate != nullptr) xt.gate = reinterpret_cast<const T*>(x.gate) + t0 * x.gate_ld;
    const cudaError_t e = launch_pdl(paged_attend_kernel<T, O, RL>, dim3(A.heads, n - t0 < 65535 ? n - t0 : 65535), dim3(128), bytes, s,
                                     q + t0 * A.q_row, kc, vc, bt, mb_, bs, seq != nullptr ? seq + t0 : seq, pos + t0, slots + t0, sink,
                                     out + t0 * A.o_row, A, xt);
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  return 0;
}

template <typename T, typename O>
static int attend(const T* q, const T* kc, const T* vc, const int* bt, int mb_, int bs, const int* seq, const int* pos, const long long* slots,
                  const T* sink, O* out, int n, MbAttend A, MbScores x, cudaStream_t s) {
  if (A.dv <= 128) return attend_rl<T, O, 4>(q, kc, vc, bt, mb_, bs, seq, pos, slots, sink, out, n, A, x, s);
  if (A.dv <= 256) return attend_rl<T, O, 8>(q, kc, vc, bt, mb_, bs, seq, pos, slots, sink, out, n, A, x, s);
  if (A.dv <= 512) return attend_rl<T, O, 16>(q, kc, vc, bt, mb_, bs, seq, pos, slots, sink, out, n, A, x, s);
  if (A.dv <= 1024) return attend_rl<T, O, 32>(q, kc, vc, bt, mb_, bs, seq, pos, slots, sink, out, n, A, x, s);
  return -3;
}

}  // namespace mx
}  // namespace mb

using namespace mb;
using namespace mb::mx;

extern "C" int mb_paged_attend(const void* q, const void* kc, const void* vc, const int* block_table, int max_blocks, int block_size,
                               const int* token_seq, const int* positions, const long long* slots, const void* sink, void* out, int T,
                               MbAttend A, MbScores x, int f32, int out_f32, cudaStream_t s) {
  if (T <= 0) return 0;
  if (A.heads <= 0 || A.group <= 0 || A.heads % A.group) return -3;
  auto run = [&](auto ty, auto to) {
    using E = decltype(ty);
    using O = decltype(to);
    return attend<E, O>(reinterpret_cast<const E*>(q), reinterpret_cast<const E*>(kc), reinterpret_cast<const E*>(vc), block_table, max_blocks,
                  block_size, token_seq, positions, slots, reinterpret_cast<const E*>(sink), reinterpret_cast<O*>(out), T, A, x, s);
  };
  if (f32) return run(float{}, float{});
  return out_f32 ? run(bf16{}, float{}) : run(bf16{}, bf16{});
}
