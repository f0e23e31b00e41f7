// What stands between a differential-attention layer's input projection [q | k | v | gate] and its attention, one launch: part 0 of a
// token's CTAs norms its queries head by head and map by map and multiplies them by the temperature of their position; part 1 does the
// same with the keys (no temperature) and writes keys and values to the paged cache; the last part is the aside of mixers.cuh.  A layer that
// reads another layer's keys and values has no part 1.
//
// A prepared query row (head h, map m) has the map's half of a key head's [map 1 | map 2] and zeros in the other half, so that the two maps
// of a head are two heads of the grouped-query kernels over the same keys and values.
//
//   diff_combine_kernel   difference, norm and gate behind the any-size attention kernel (the tensor-core kernels do it themselves)
#include "mixers.cuh"

namespace mb {
namespace mx {

static constexpr int kDiff = 256;

// `rows` rows of `dim` values x → y(row): x / rms(x) · w · mul.  A row is normed by `lanes` neighbouring lanes (VEC: one 16-byte piece
// each, a power of two of them) or by a warp.
template <typename T, bool VEC, typename F>
__device__ __forceinline__ void norm_rows(const T* __restrict__ x, const T* __restrict__ w, int rows, int dim, float eps, float mul, F&& y) {
  constexpr int V = 16 / static_cast<int>(sizeof(T));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if constexpr (VEC) {
    const int pieces = dim / V;
    int lanes = 1;
    while (lanes < pieces) lanes *= 2;                   // ≤ 32 (checked by the launcher)
    const int per = 32 / lanes, sub = lane / lanes, c = (lane % lanes) * V;
    const bool on = c < dim;
    float g[V];
    if (on) load_n<V>(w + c, g);
    for (int r0 = warp * per; r0 < rows; r0 += (kDiff / 32) * per) {
      const int r = r0 + sub;
      float f[V], ss = 0.f;
      if (on && r < rows) {
        load_n<V>(x + static_cast<long long>(r) * dim + c, f);
#pragma unroll
        for (int j = 0; j < V; ++j) ss = fmaf(f[j], f[j], ss);
      }
      for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float s = rsqrt_exact(__fdiv_rn(ss, static_cast<float>(dim)) + eps) * mul;
      if (on && r < rows) {
#pragma unroll
        for (int j = 0; j < V; ++j) f[j] = f[j] * s * g[j];
        store_n<V>(y(r) + c, f);
      }
    }
  } else {
    for (int r = warp; r < rows; r += kDiff / 32) {
      const T* xr = x + static_cast<long long>(r) * dim;
      float ss = 0.f;
      for (int c = lane; c < dim; c += 32) ss = fmaf(to_f(xr[c]), to_f(xr[c]), ss);
      const float s = rsqrt_exact(__fdiv_rn(warp_sum(ss), static_cast<float>(dim)) + eps) * mul;
      for (int c = lane; c < dim; c += 32) y(r)[c] = from_f<T>(to_f(xr[c]) * s * to_f(w[c]));
    }
  }
}

template <typename T, bool VEC, bool GROUPED>
__global__ void __launch_bounds__(kDiff) diff_prep_kernel(const T* __restrict__ proj, long long ld, const int* __restrict__ positions,
                                                          const long long* __restrict__ slots, const T* __restrict__ q_norm,
                                                          const T* __restrict__ k_norm, const T* __restrict__ lvec, float* __restrict__ lam,
                                                          T* __restrict__ kc, T* __restrict__ vc, T* __restrict__ q, MbDiffPrep L, MbAside a) {
  pdl_trigger();
  pdl_wait();
  constexpr int V = VEC ? 16 / static_cast<int>(sizeof(T)) : 1;
  const long long t = blockIdx.x;
  const T* p = proj + t * ld;
  const int nq = L.heads * 2 * L.dim, nk = L.kv_heads * 2 * L.dim, nv = L.kv_heads * L.vdim;
  if (blockIdx.y == (L.kv_heads > 0 ? 2 : 1)) {
    aside_row<T, VEC, kDiff, GROUPED>(a, t);
    return;
  }
  if (blockIdx.y == 0) {
    if (t == 0 && threadIdx.x >= kDiff - 32) {          // the weight of the second map, one number for the layer
      const int lane = threadIdx.x & 31;
      float s1 = 0.f, s2 = 0.f;
      for (int c = lane; c < L.dim; c += 32) {
        s1 = fmaf(to_f(lvec[c]), to_f(lvec[L.dim + c]), s1);
        s2 = fmaf(to_f(lvec[2 * L.dim + c]), to_f(lvec[3 * L.dim + c]), s2);
      }
      s1 = warp_sum(s1);
      s2 = warp_sum(s2);
      if (lane == 0) *lam = exp_t<T>(s1) - exp_t<T>(s2) + L.diff;
    }
    float mul = 1.f;
    if (L.temp_coef != 0.f) mul += L.temp_coef * static_cast<float>(log(floor((positions[t] + 1.0) / L.temp_every) + 1.0));
    T* y = q + t * L.heads * 2 * L.q_pitch;
    norm_rows<T, VEC>(p, q_norm, 2 * L.heads, L.dim, L.eps, mul, [&](int r) { return y + static_cast<long long>(r) * L.q_pitch + (r & 1) * L.dim; });
    const int rest = L.q_pitch - L.dim;                 // the other map's half and the padding
    for (int i = threadIdx.x * V; i < 2 * L.heads * rest; i += kDiff * V) {
      const int r = i / rest, c = i - r * rest;
      float z[V];
#pragma unroll
      for (int j = 0; j < V; ++j) z[j] = 0.f;
      store_n<V>(y + static_cast<long long>(r) * L.q_pitch + ((r & 1) && c < L.dim ? c : c + L.dim), z);
    }
    return;
  }
  const long long slot = slots[t];
  if (slot < 0) return;                                 // padding row of a decode batch
  T* k = kc + slot * nk;
  norm_rows<T, VEC>(p + nq, k_norm, 2 * L.kv_heads, L.dim, L.eps, 1.f, [&](int r) { return k + static_cast<long long>(r) * L.dim; });
  T* v = vc + slot * nv;
  for (int i = threadIdx.x * V; i < nv; i += kDiff * V) {
    float f[V];
    load_n<V>(p + nq + nk + i, f);
    store_n<V>(v + i, f);
  }
}

// a warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) diff_combine_kernel(const float* __restrict__ a, T* __restrict__ out, long long o_row, long long n, int heads,
                                                           int vdim, MbDiff d) {
  pdl_trigger();
  pdl_wait();
  const long long i = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (i >= n) return;
  const long long t = i / heads;
  const int h = static_cast<int>(i - t * heads);
  const float* a1 = a + i * 2 * vdim;
  const float* a2 = a1 + vdim;
  const float lam = *d.lam;
  float ss = 0.f;
  for (int c = lane; c < vdim; c += 32) {
    const float o = fmaf(-lam, a2[c], a1[c]);
    ss = fmaf(o, o, ss);
  }
  const float rstd = rsqrt_exact(__fdiv_rn(warp_sum(ss), static_cast<float>(vdim)) + d.eps);
  const float f = rstd * d.gain * sigmoid_t<T>(to_f(reinterpret_cast<const T*>(d.gate)[t * d.gate_ld + h]));
  for (int c = lane; c < vdim; c += 32) out[t * o_row + static_cast<long long>(h) * vdim + c] = from_f<T>(fmaf(-lam, a2[c], a1[c]) * f);
}

}  // namespace mx
}  // namespace mb

using namespace mb;
using namespace mb::mx;

extern "C" int mb_diff_prep(const void* proj, long long ld, const int* positions, const long long* slots, const void* q_norm, const void* k_norm,
                            const void* lvec, float* lam, void* kc, void* vc, void* q, int T, MbDiffPrep L, MbAside a, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  if (L.heads <= 0 || L.dim <= 0 || L.q_pitch < 2 * L.dim || !aside_ok(a)) return -3;
  auto run = [&](auto ty) {
    using E = decltype(ty);
    constexpr int v = 16 / static_cast<int>(sizeof(E));
    const bool vec = ld % v == 0 && L.dim % v == 0 && L.dim <= 32 * v && L.vdim % v == 0 && L.q_pitch % v == 0 &&
                     (reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q)) % 16 == 0 && aside_vec<E>(a);
    auto kern = a.grouped ? (vec ? diff_prep_kernel<E, true, true> : diff_prep_kernel<E, false, true>)
                          : (vec ? diff_prep_kernel<E, true, false> : diff_prep_kernel<E, false, false>);
    return static_cast<int>(launch_pdl(kern, dim3(T, (L.kv_heads > 0 ? 2 : 1) + aside_on(a)), dim3(kDiff), 0, s, reinterpret_cast<const E*>(proj), ld,
                                       positions, slots, reinterpret_cast<const E*>(q_norm), reinterpret_cast<const E*>(k_norm),
                                       reinterpret_cast<const E*>(lvec), lam, reinterpret_cast<E*>(kc), reinterpret_cast<E*>(vc),
                                       reinterpret_cast<E*>(q), L, a));
  };
  return f32 ? run(float{}) : run(bf16{});
}

extern "C" int mb_diff_combine(const float* a, void* out, long long o_row, int T, int heads, int vdim, MbDiff d, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  const long long n = static_cast<long long>(T) * heads;
  auto run = [&](auto ty) {
    using E = decltype(ty);
    return static_cast<int>(launch_pdl(diff_combine_kernel<E>, dim3(static_cast<unsigned>((n + 7) / 8)), dim3(256), 0, s, a, reinterpret_cast<E*>(out), o_row,
                                       n, heads, vdim, d));
  };
  return f32 ? run(float{}) : run(bf16{});
}
