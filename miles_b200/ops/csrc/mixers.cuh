// Shared device helpers of the layer-by-layer decoder kernels (mixers.cu, latent_attn.cu, linear_state.cu).
//
// Those kernels are templates over the model's dtype T.  With T = float the result must be good to 32 bits although the
// extension is compiled with fast math, so exponentials go through double precision and divisions and roots use the
// correctly rounded intrinsics; with T = bf16 the fast forms are used.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "launch.h"
#include "pdl.cuh"

namespace mb {
namespace mx {

using bf16 = __nv_bfloat16;

template <typename T> struct is_exact { static constexpr bool value = false; };
template <> struct is_exact<float> { static constexpr bool value = true; };

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16(v); }

template <typename T> __device__ __forceinline__ float exp_t(float x) {
  if constexpr (is_exact<T>::value) return static_cast<float>(exp(static_cast<double>(x)));
  else return __expf(x);
}
template <typename T> __device__ __forceinline__ float sigmoid_t(float x) {
  if constexpr (is_exact<T>::value) return static_cast<float>(1.0 / (1.0 + exp(-static_cast<double>(x))));
  else return __fdividef(1.f, 1.f + __expf(-x));
}
// __fdividef(1, inf) is 0 and __expf(88.8…) is inf, so sigmoid_t(−large) is 0 as it should be
template <typename T> __device__ __forceinline__ float silu_t(float x) { return x * sigmoid_t<T>(x); }
__device__ __forceinline__ float rsqrt_exact(float x) { return __fdiv_rn(1.f, __fsqrt_rn(x)); }

template <typename T> __device__ __forceinline__ float softplus_t(float x) {
  if constexpr (is_exact<T>::value) {
    const double d = x;
    return static_cast<float>(d > 0. ? d + log1p(exp(-d)) : log1p(exp(d)));
  } else {
    const float e = __expf(-fabsf(x));
    return fmaxf(x, 0.f) + log1pf(e);
  }
}

// N consecutive values ↔ floats (N·sizeof(T) bytes, 16-byte aligned pieces)
template <int N> __device__ __forceinline__ void load_n(const float* p, float (&f)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 4) {
      const float4 v = *reinterpret_cast<const float4*>(p + i);
      f[i] = v.x; f[i + 1] = v.y; f[i + 2] = v.z; f[i + 3] = v.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = p[i];
  }
}
template <int N> __device__ __forceinline__ void load_n(const bf16* p, float (&f)[N]) {
  if constexpr (N == 8) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = __uint_as_float(w[i] << 16);
      f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = __bfloat162float(p[i]);
  }
}
template <int N> __device__ __forceinline__ void store_n(float* p, const float (&f)[N]) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) p[i] = f[i];
  }
}
template <int N> __device__ __forceinline__ void store_n(bf16* p, const float (&f)[N]) {
  if constexpr (N == 8) {
    uint32_t w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      __nv_bfloat162 h = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
      w[i] = *reinterpret_cast<uint32_t*>(&h);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) p[i] = __float2bfloat16(f[i]);
  }
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
template <int THREADS>
__device__ __forceinline__ float block_sum(float v, float* sh) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
  __syncthreads();
  float r = 0.f;
#pragma unroll
  for (int w = 0; w < THREADS / 32; ++w) r += sh[w];
  return r;
}

// cs[0 … half) = cosines, cs[half … 2·half) = sines of position · frequency, times `magnitude`; angles in double precision, so that a
// position of any size costs no accuracy.  The caller's CTA barrier comes after.
template <typename T, int THREADS>
__device__ __forceinline__ void rotary_table(float* cs, int position, const double* __restrict__ freq, int half, float magnitude) {
  const double pos = position;
  for (int i = threadIdx.x; i < half; i += THREADS) {
    double a = pos * freq[i];
    a -= rint(a * 0.15915494309189535) * 6.283185307179586;      // one turn off per whole turn: |a| ≤ π
    if constexpr (is_exact<T>::value) {
      double s, c;
      sincos(a, &s, &c);
      cs[i] = static_cast<float>(c * magnitude);
      cs[half + i] = static_cast<float>(s * magnitude);
    } else {
      float s, c;
      __sincosf(static_cast<float>(a), &s, &c);
      cs[i] = c * magnitude;
      cs[half + i] = s * magnitude;
    }
  }
}

// gate · sigmoid(alpha · gate) · (up + shift) with gate ≤ limit and |up| ≤ limit (limit ∞, alpha 1, shift 0: silu(gate) · up)
template <typename T> __device__ __forceinline__ float clamped_glu_t(float gate, float up, float limit, float alpha, float shift) {
  const float a = fminf(gate, limit), b = fminf(fmaxf(up, -limit), limit);
  return a * sigmoid_t<T>(alpha * a) * (b + shift);
}
__device__ __forceinline__ float relu_square(float v) { v = fmaxf(v, 0.f); return v * v; }

// A float's bits in an order that integers compare: larger float, larger key.  NaN: 0, below everything.
__device__ __forceinline__ uint32_t order_key(float v) {
  const uint32_t b = __float_as_uint(v);
  if ((b & 0x7fffffffu) > 0x7f800000u) return 0u;
  if (b == 0x80000000u) return 0x80000000u;                // −0 is 0
  return (b & 0x80000000u) ? ~b : b | 0x80000000u;
}
__device__ __forceinline__ float key_value(uint32_t k) { return __uint_as_float((k & 0x80000000u) ? k & 0x7fffffffu : ~k); }

// One warp chooses the K largest of E logits (ties: the lower index) and weighs them by a softmax over the chosen ones.  A row of
// NaNs leaves index −1, weight 0.  Up to 32 · kLocal logits stay in registers; more are read again for every choice.
template <typename T>
__device__ __forceinline__ void topk_softmax_row(const float* __restrict__ z, int E, int K, float* __restrict__ w, int* __restrict__ idx) {
  constexpr int kLocal = 8;
  const int lane = threadIdx.x & 31;
  const bool local = E <= 32 * kLocal;
  uint32_t key[kLocal];
#pragma unroll
  for (int i = 0; i < kLocal; ++i) key[i] = i * 32 + lane < E ? order_key(z[i * 32 + lane]) : 0u;
  uint32_t last = 0xffffffffu;
  int last_i = -1;
  float first = 0.f, sum = 0.f;
  for (int j = 0; j < K; ++j) {
    uint32_t bk = 0u;
    int bi = 0x7fffffff;
    if (local) {
#pragma unroll
      for (int i = 0; i < kLocal; ++i)
        if (key[i] > bk) { bk = key[i]; bi = i * 32 + lane; }      // ascending index: ties keep the lower one
    } else {
      for (int e = lane; e < E; e += 32) {
        const uint32_t k = order_key(z[e]);
        if ((k < last || (k == last && e > last_i)) && k > bk) { bk = k; bi = e; }
      }
    }
    const uint32_t top = __reduce_max_sync(0xffffffffu, bk);
    const int at = __reduce_min_sync(0xffffffffu, bk == top ? bi : 0x7fffffff);
    const bool found = top != 0u;
    const float v = key_value(top);
    if (j == 0) first = v;
    const float p = found ? exp_t<T>(v - first) : 0.f;
    sum += p;
    if (lane == (j & 31)) { idx[j] = found ? at : -1; w[j] = p; }
    if (local && (at & 31) == lane) {
#pragma unroll
      for (int i = 0; i < kLocal; ++i)
        if (i * 32 + lane == at) key[i] = 0u;
    }
    last = top;
    last_i = at;
  }
  for (int j = lane; j < K; j += 32) w[j] = sum > 0.f ? __fdiv_rn(w[j], sum) : 0.f;      // every lane reads back what it wrote
}

// One warp chooses the K largest of E choice scores σ(z) + correction among the experts of the `keep` best of `groups` equal groups of
// neighbours (a group is worth the sum of its two largest choice scores), ties to the lower index, and weighs the chosen ones by their
// σ(z) over the sum of those, times `scale`.  Index −1 with weight 0 where nothing is left to choose (NaNs).  groups ≤ 256.
template <typename T>
__device__ __forceinline__ void topk_grouped_row(const float* __restrict__ z, const T* __restrict__ correction, int E, int K, int groups, int keep,
                                                 float scale, float* __restrict__ w, int* __restrict__ idx) {
  constexpr int kLocal = 8;                      // keys (and groups) per lane that stay in registers
  const int lane = threadIdx.x & 31, size = E / groups;
  const bool local = E <= 32 * kLocal;
  auto key_of = [&](int e) -> uint32_t { return order_key(sigmoid_t<T>(z[e]) + (correction != nullptr ? to_f(correction[e]) : 0.f)); };
  uint32_t key[kLocal], open[kLocal];            // open: bit g of the groups whose experts can be chosen
#pragma unroll
  for (int i = 0; i < kLocal; ++i) {
    key[i] = local && i * 32 + lane < E ? key_of(i * 32 + lane) : 0u;
    open[i] = 0xffffffffu;
  }
  if (keep < groups) {
    uint32_t worth[kLocal];                      // of group i·32 + lane
#pragma unroll
    for (int i = 0; i < kLocal; ++i) { worth[i] = 0u; open[i] = 0u; }
    for (int g = 0; g < groups; ++g) {
      uint32_t b1 = 0u, b2 = 0u;                 // the lane's two largest of the group
      auto see = [&](uint32_t k) {
        if (k > b1) { b2 = b1; b1 = k; }
        else if (k > b2) b2 = k;
      };
      if (local) {
#pragma unroll
        for (int i = 0; i < kLocal; ++i) {
          const int e = i * 32 + lane;
          if (e >= g * size && e < (g + 1) * size) see(key[i]);
        }
      } else {
        for (int e = g * size + lane; e < (g + 1) * size; e += 32) see(key_of(e));
      }
      const uint32_t top = __reduce_max_sync(0xffffffffu, b1);
      const int owner = __ffs(__ballot_sync(0xffffffffu, b1 == top)) - 1;
      const uint32_t second = __reduce_max_sync(0xffffffffu, lane == owner ? b2 : b1);
      const uint32_t v = top == 0u ? 0u : order_key(key_value(top) + (second != 0u ? key_value(second) : 0.f));
#pragma unroll
      for (int i = 0; i < kLocal; ++i)
        if (i * 32 + lane == g) worth[i] = v;
    }
    for (int j = 0; j < keep; ++j) {
      uint32_t bk = 0u;
      int bi = 0x7fffffff;
#pragma unroll
      for (int i = 0; i < kLocal; ++i)
        if (worth[i] > bk) { bk = worth[i]; bi = i * 32 + lane; }
      const uint32_t top = __reduce_max_sync(0xffffffffu, bk);
      if (top == 0u) break;
      const int at = __reduce_min_sync(0xffffffffu, bk == top ? bi : 0x7fffffff);
#pragma unroll
      for (int i = 0; i < kLocal; ++i) {
        if (i * 32 + lane == at) worth[i] = 0u;
        if ((at >> 5) == i) open[i] |= 1u << (at & 31);
      }
    }
  }
  auto is_open = [&](int e) -> bool {
    const int g = e / size;
    bool r = false;
#pragma unroll
    for (int i = 0; i < kLocal; ++i)
      if ((g >> 5) == i) r = (open[i] >> (g & 31)) & 1u;
    return r;
  };
  if (keep < groups && local) {
#pragma unroll
    for (int i = 0; i < kLocal; ++i)
      if (i * 32 + lane < E && !is_open(i * 32 + lane)) key[i] = 0u;
  }
  uint32_t last = 0xffffffffu;
  int last_i = -1;
  float sum = 0.f;
  for (int j = 0; j < K; ++j) {
    uint32_t bk = 0u;
    int bi = 0x7fffffff;
    if (local) {
#pragma unroll
      for (int i = 0; i < kLocal; ++i)
        if (key[i] > bk) { bk = key[i]; bi = i * 32 + lane; }
    } else {
      for (int e = lane; e < E; e += 32) {
        const uint32_t k = is_open(e) ? key_of(e) : 0u;
        if ((k < last || (k == last && e > last_i)) && k > bk) { bk = k; bi = e; }
      }
    }
    const uint32_t top = __reduce_max_sync(0xffffffffu, bk);
    const int at = __reduce_min_sync(0xffffffffu, bk == top ? bi : 0x7fffffff);
    const bool found = top != 0u;
    const float s = found ? sigmoid_t<T>(z[at]) : 0.f;
    sum += s;
    if (lane == (j & 31)) { idx[j] = found ? at : -1; w[j] = s; }
    if (local && found && (at & 31) == lane) {
#pragma unroll
      for (int i = 0; i < kLocal; ++i)
        if (i * 32 + lane == at) key[i] = 0u;
    }
    last = top;
    last_i = at;
  }
  for (int j = lane; j < K; j += 32) w[j] = __fdiv_rn(w[j], sum + 1e-20f) * scale;      // every lane reads back what it wrote
}

// What runs beside a mixer's preparation for token t, by a CTA of THREADS threads: its choice of experts and the activation of its
// dense feed-forward (see MbAside).  GROUPED: the kernel holds the choice among groups instead of the softmax one.
template <typename T, bool VEC, int THREADS, bool GROUPED>
__device__ __forceinline__ void aside_row(const MbAside& a, long long t) {
  if (a.logits != nullptr && threadIdx.x < 32) {
    if constexpr (GROUPED)
      topk_grouped_row<T>(a.logits + t * a.experts, reinterpret_cast<const T*>(a.correction), a.experts, a.top, a.groups, a.keep, a.scale,
                          a.weights + t * a.top, a.index + t * a.top);
    else
      topk_softmax_row<T>(a.logits + t * a.experts, a.experts, a.top, a.weights + t * a.top, a.index + t * a.top);
  }
  if (a.glu_in == nullptr) return;
  const T* in = reinterpret_cast<const T*>(a.glu_in) + t * a.glu_ld_in;
  T* out = reinterpret_cast<T*>(a.glu_out) + t * a.glu_ld_out;
  constexpr int V = VEC ? 16 / static_cast<int>(sizeof(T)) : 1;
  for (int i = threadIdx.x * V; i < a.ff; i += THREADS * V) {
    float g[V], u[V];
    load_n<V>(in + i, g);
    load_n<V>(in + a.ff + i, u);
#pragma unroll
    for (int j = 0; j < V; ++j) g[j] = clamped_glu_t<T>(g[j], u[j], a.limit, a.alpha, a.shift);
    store_n<V>(out + i, g);
  }
}
// 16-byte accesses fit the feed-forward of an aside
template <typename T>
inline bool aside_vec(const MbAside& a) {
  constexpr int v = 16 / static_cast<int>(sizeof(T));
  return a.glu_in == nullptr || (a.ff % v == 0 && a.glu_ld_in % v == 0 && a.glu_ld_out % v == 0 &&
                                 (reinterpret_cast<uintptr_t>(a.glu_in) | reinterpret_cast<uintptr_t>(a.glu_out)) % 16 == 0);
}
inline bool aside_on(const MbAside& a) { return a.logits != nullptr || a.glu_in != nullptr; }
inline bool aside_ok(const MbAside& a) {
  return a.logits == nullptr || !a.grouped || (a.groups > 0 && a.groups <= 256 && a.experts % a.groups == 0 && a.keep > 0);
}

}  // namespace mx
}  // namespace mb
