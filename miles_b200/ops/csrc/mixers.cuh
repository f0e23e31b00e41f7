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

// gate · sigmoid(alpha · gate) · (up + 1) with gate ≤ limit and |up| ≤ limit
template <typename T> __device__ __forceinline__ float clamped_glu_t(float gate, float up, float limit, float alpha) {
  const float a = fminf(gate, limit), b = fminf(fmaxf(up, -limit), limit);
  return a * sigmoid_t<T>(alpha * a) * (b + 1.f);
}

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

}  // namespace mx
}  // namespace mb
