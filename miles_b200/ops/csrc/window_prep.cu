// What stands between a grouped-query layer's input projection and its attention, one launch: CTA (token, 0) norms a token's whole
// query projection and rotates its heads; the next one, for a layer with keys and values of its own, does the same with the keys and
// writes keys and values (over their root mean square per head, if asked for) to the paged cache; the last one, if there is any,
// chooses the token's experts and applies the activation of the dense feed-forward that shares the projection.  fp32 math in every
// dtype T.
#include "mixers.cuh"

namespace mb {
namespace mx {

static constexpr int kPrep = 256;

template <typename T, bool VEC>
__device__ __forceinline__ float square_sum(const T* __restrict__ x, int n, float* sh) {
  constexpr int V = VEC ? 16 / static_cast<int>(sizeof(T)) : 1;
  float ss = 0.f;
#pragma unroll 2
  for (int i = threadIdx.x * V; i < n; i += kPrep * V) {
    float a[V];
    load_n<V>(x + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += a[j] * a[j];
  }
  return block_sum<kPrep>(ss, sh);
}

// heads × dim values x → y (`pitch` per head, zeros behind dim): x · rstd · w, the first `rot` of every head rotated in pairs
template <typename T, bool VEC>
__device__ __forceinline__ void norm_rotate(const T* __restrict__ x, const T* __restrict__ w, float rstd, const float* cs, T* __restrict__ y,
                                            int heads, int dim, int rot, int pitch) {
  const int half = rot / 2;
  if constexpr (VEC) {
    constexpr int V = 16 / static_cast<int>(sizeof(T));
    const int n = dim / V;
#pragma unroll 2
    for (int i = threadIdx.x; i < heads * n; i += kPrep) {
      const int h = i / n, c = (i - h * n) * V;
      float f[V], g[V];
      load_n<V>(x + i * V, f);
      if (w != nullptr) {
        load_n<V>(w + i * V, g);
#pragma unroll
        for (int j = 0; j < V; ++j) f[j] *= rstd * g[j];
      }
      if (c < rot) {
#pragma unroll
        for (int j = 0; j < V; j += 2) {
          const float u = f[j], v = f[j + 1], co = cs[(c + j) >> 1], si = cs[half + ((c + j) >> 1)];
          f[j] = u * co - v * si;
          f[j + 1] = v * co + u * si;
        }
      }
      store_n<V>(y + h * pitch + c, f);
    }
  } else {
    for (int i = threadIdx.x; i < heads * dim; i += kPrep) {
      const int h = i / dim, c = i - h * dim;
      auto at = [&](int k) { return to_f(x[k]) * (w != nullptr ? rstd * to_f(w[k]) : 1.f); };
      float f = at(i);
      if (c < rot) {
        const float co = cs[c >> 1], si = cs[half + (c >> 1)];
        f = (c & 1) ? f * co + at(i - 1) * si : f * co - at(i + 1) * si;
      }
      y[h * pitch + c] = from_f<T>(f);
    }
  }
  const int gap = pitch - dim;
  for (int i = threadIdx.x; i < heads * gap; i += kPrep) y[(i / gap) * pitch + dim + i % gap] = from_f<T>(0.f);
}

template <typename T, bool VEC, bool GROUPED>
__global__ void __launch_bounds__(kPrep) window_prep_kernel(const T* __restrict__ proj, long long ld, const int* __restrict__ positions,
                                                            const long long* __restrict__ slots, const double* __restrict__ freq,
                                                            float magnitude, const T* __restrict__ q_norm, const T* __restrict__ k_norm, int v_norm,
                                                            float eps, T* __restrict__ kc, T* __restrict__ vc, T* __restrict__ q, MbWindow L,
                                                            MbAside a) {
  extern __shared__ float cs[];          // [rot/2] cosines, [rot/2] sines
  __shared__ float sh[kPrep / 32];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const T* p = proj + t * ld;
  const int nq = L.heads * L.dim, nk = L.kv_heads * L.dim, nv = L.kv_heads * L.vdim;
  const int role = blockIdx.y + (kc == nullptr && blockIdx.y > 0 ? 1 : 0);
  if (role == 2) {
    aside_row<T, VEC, kPrep, GROUPED>(a, t);
    return;
  }
  const bool keys = role == 1;
  const long long slot = slots[t];
  if (keys && slot < 0) return;          // padding row of a decode batch
  rotary_table<T, kPrep>(cs, positions[t], freq, L.rot / 2, magnitude);
  const T* x = keys ? p + nq : p;
  const T* w = keys ? k_norm : q_norm;
  const int n = keys ? nk : nq;
  float rstd = 1.f;
  if (w != nullptr) rstd = rsqrt_exact(__fdiv_rn(square_sum<T, VEC>(x, n, sh), static_cast<float>(n)) + eps);
  __syncthreads();
  if (!keys) {
    norm_rotate<T, VEC>(x, w, rstd, cs, q + t * L.heads * static_cast<long long>(L.q_pitch), L.heads, L.dim, L.rot, L.q_pitch);
    return;
  }
  norm_rotate<T, VEC>(x, w, rstd, cs, kc + slot * nk, L.kv_heads, L.dim, L.rot, L.dim);
  constexpr int V = VEC ? 16 / static_cast<int>(sizeof(T)) : 1;
  T* v = vc + slot * nv;
  if (v_norm) {                          // a warp per head
    const int lane = threadIdx.x & 31;
    for (int h = threadIdx.x >> 5; h < L.kv_heads; h += kPrep / 32) {
      const T* xv = p + nq + nk + h * L.vdim;
      float f[V], ss = 0.f;
      for (int i = lane * V; i < L.vdim; i += 32 * V) {
        load_n<V>(xv + i, f);
#pragma unroll
        for (int j = 0; j < V; ++j) ss += f[j] * f[j];
      }
      const float r = rsqrt_exact(__fdiv_rn(warp_sum(ss), static_cast<float>(L.vdim)) + eps);
      for (int i = lane * V; i < L.vdim; i += 32 * V) {
        load_n<V>(xv + i, f);
#pragma unroll
        for (int j = 0; j < V; ++j) f[j] *= r;
        store_n<V>(v + h * L.vdim + i, f);
      }
    }
    return;
  }
  for (int i = threadIdx.x * V; i < nv; i += kPrep * V) {
    float f[V];
    load_n<V>(p + nq + nk + i, f);
    store_n<V>(v + i, f);
  }
}

template <typename T>
static int prep(const T* proj, long long ld, const int* positions, const long long* slots, const double* freq, float magnitude,
                const T* q_norm, const T* k_norm, int v_norm, float eps, T* kc, T* vc, T* q, int n, MbWindow L, MbAside a, cudaStream_t s) {
  const int v = 16 / static_cast<int>(sizeof(T));
  const bool vec = ld % v == 0 && L.dim % v == 0 && L.vdim % v == 0 && L.rot % v == 0 && L.q_pitch % v == 0 && reinterpret_cast<uintptr_t>(proj) % 16 == 0 && aside_vec<T>(a);
  auto kern = a.grouped ? (vec ? window_prep_kernel<T, true, true> : window_prep_kernel<T, false, true>)
                        : (vec ? window_prep_kernel<T, true, false> : window_prep_kernel<T, false, false>);
  return static_cast<int>(launch_pdl(kern, dim3(n, 1 + (kc != nullptr) + aside_on(a)), dim3(kPrep), L.rot * sizeof(float), s, proj,
                                     ld, positions, slots, freq, magnitude, q_norm, k_norm, v_norm, eps, kc, vc, q, L, a));
}

}  // namespace mx
}  // namespace mb

using namespace mb;
using namespace mb::mx;

extern "C" int mb_window_prep(const void* proj, long long ld, const int* positions, const long long* slots, const double* freq,
                              float magnitude, const void* q_norm, const void* k_norm, int v_norm, float eps, void* kc, void* vc, void* q, int T,
                              MbWindow L, MbAside a, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  if (L.rot > 4096 || L.rot % 2 || L.rot > L.dim || L.heads % L.kv_heads || !aside_ok(a)) return -3;
  auto run = [&](auto ty) {
    using E = decltype(ty);
    return prep(reinterpret_cast<const E*>(proj), ld, positions, slots, freq, magnitude, reinterpret_cast<const E*>(q_norm),
                reinterpret_cast<const E*>(k_norm), v_norm, eps, reinterpret_cast<E*>(kc), reinterpret_cast<E*>(vc), reinterpret_cast<E*>(q), T, L, a, s);
  };
  return f32 ? run(float{}) : run(bf16{});
}
