// Row-wise kernels of the layer-by-layer decoders: hashed-bigram embedding, output norm + layer scale + fp32 residual (with the
// model's final norm fused into the last one), clamped gated activation, gated norm over all heads of a mixer.
// fp32 math; activations in the model's dtype T (bf16, or float for 32-bit runs).
#include <type_traits>

#include "mixers.cuh"

namespace mb {
namespace mx {

static constexpr int kRow = 256;

// x[t] = embed[tok] + table[(prev·mul_prev + tok·mul_cur) mod buckets]; the last row of the table for a sequence's first token
template <typename T, int V>
__global__ void __launch_bounds__(128) bigram_embed_kernel(const int* __restrict__ tok, const int* __restrict__ prev,
                                                           const T* __restrict__ embed, const T* __restrict__ table, long long buckets,
                                                           long long mul_prev, long long mul_cur, float* __restrict__ x,
                                                           T* __restrict__ xb, int D) {
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const long long id = tok[t];
  long long row = 0;
  if (table != nullptr) {
    const long long p = prev[t];
    row = p < 0 ? buckets : (p * mul_prev + id * mul_cur) % buckets;
  }
  for (int i = threadIdx.x * V; i < D; i += 128 * V) {
    float a[V];
    load_n<V>(embed + id * D + i, a);
    if (table != nullptr) {
      float b[V];
      load_n<V>(table + row * D + i, b);
#pragma unroll
      for (int j = 0; j < V; ++j) a[j] += b[j];
    }
    store_n<V>(x + t * D + i, a);
    store_n<V>(xb + t * D + i, a);
  }
}

// x += y / rms(y) · nw · ls;  xb = x, or x / rms(x) · fw with the model's final norm
template <typename T, int V>
__global__ void __launch_bounds__(kRow) output_norm_kernel(float* __restrict__ x, const T* __restrict__ y, const T* __restrict__ nw,
                                                           const T* __restrict__ ls, const T* __restrict__ fw, T* __restrict__ xb, int D,
                                                           float eps) {
  __shared__ float sh[kRow / 32];
  pdl_trigger();
  pdl_wait();
  const long long base = static_cast<long long>(blockIdx.x) * D;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < D; i += kRow * V) {
    float a[V];
    load_n<V>(y + base + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += a[j] * a[j];
  }
  const float rstd = rsqrt_exact(__fdiv_rn(block_sum<kRow>(ss, sh), static_cast<float>(D)) + eps);
  ss = 0.f;
  for (int i = threadIdx.x * V; i < D; i += kRow * V) {
    float a[V], w[V], l[V], r[V];
    load_n<V>(y + base + i, a);
    load_n<V>(nw + i, w);
    load_n<V>(ls + i, l);
    load_n<V>(x + base + i, r);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      r[j] += a[j] * rstd * w[j] * l[j];
      ss += r[j] * r[j];
    }
    store_n<V>(x + base + i, r);
    if (fw == nullptr) store_n<V>(xb + base + i, r);
  }
  if (fw == nullptr) return;
  const float rs2 = rsqrt_exact(__fdiv_rn(block_sum<kRow>(ss, sh), static_cast<float>(D)) + eps);
  for (int i = threadIdx.x * V; i < D; i += kRow * V) {      // every thread reads back what it wrote itself
    float w[V], r[V];
    load_n<V>(fw + i, w);
    load_n<V>(x + base + i, r);
#pragma unroll
    for (int j = 0; j < V; ++j) r[j] = r[j] * rs2 * w[j];
    store_n<V>(xb + base + i, r);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256) clamped_glu_kernel(const T* __restrict__ in, T* __restrict__ out, long long n_vec, int F, float limit,
                                                          float alpha) {
  pdl_trigger();
  pdl_wait();
  const int per = F / V;
  for (long long v = blockIdx.x * 256ll + threadIdx.x; v < n_vec; v += gridDim.x * 256ll) {
    const long long t = v / per;
    const int i = static_cast<int>(v - t * per) * V;
    float g[V], u[V];
    load_n<V>(in + t * 2 * F + i, g);
    load_n<V>(in + t * 2 * F + F + i, u);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float a = fminf(g[j], limit), b = fminf(fmaxf(u[j], -limit), limit);
      g[j] = a * sigmoid_t<T>(alpha * a) * (b + 1.f);
    }
    store_n<V>(out + t * F + i, g);
  }
}

// out = o / rms(o) · w · sigmoid(gate) over all C = heads · vdim channels of a token
template <typename T, int V>
__global__ void __launch_bounds__(kRow) gated_norm_kernel(const T* __restrict__ o, const T* __restrict__ w, const T* __restrict__ gate,
                                                          long long gate_ld, T* __restrict__ out, int C, float eps) {
  __shared__ float sh[kRow / 32];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < C; i += kRow * V) {
    float a[V];
    load_n<V>(o + t * C + i, a);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += a[j] * a[j];
  }
  const float rstd = rsqrt_exact(__fdiv_rn(block_sum<kRow>(ss, sh), static_cast<float>(C)) + eps);
  for (int i = threadIdx.x * V; i < C; i += kRow * V) {
    float a[V], b[V], g[V];
    load_n<V>(o + t * C + i, a);
    load_n<V>(w + i, b);
    load_n<V>(gate + t * gate_ld + i, g);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] = a[j] * rstd * b[j] * sigmoid_t<T>(g[j]);
    store_n<V>(out + t * C + i, a);
  }
}

// 16-byte accesses need element counts (and strides) that are whole vectors
template <typename F>
static int dispatch(int f32, bool vec, F&& f) {
  if (f32) return vec ? f(float{}, std::integral_constant<int, 4>{}) : f(float{}, std::integral_constant<int, 1>{});
  return vec ? f(bf16{}, std::integral_constant<int, 8>{}) : f(bf16{}, std::integral_constant<int, 1>{});
}

}  // namespace mx
}  // namespace mb

using namespace mb;
using namespace mb::mx;

extern "C" int mb_bigram_embedding(const int* tok, const int* prev, const void* embed, const void* table, long long buckets,
                                   long long mul_prev, long long mul_cur, float* x, void* xb, int T, int D, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  return dispatch(f32, D % 8 == 0, [&](auto ty, auto v) {
    using E = decltype(ty);
    return static_cast<int>(launch_pdl(bigram_embed_kernel<E, decltype(v)::value>, dim3(T), dim3(128), 0, s, tok, prev,
                                       reinterpret_cast<const E*>(embed), reinterpret_cast<const E*>(table), buckets, mul_prev, mul_cur, x,
                                       reinterpret_cast<E*>(xb), D));
  });
}

extern "C" int mb_output_norm(float* x, const void* y, const void* nw, const void* ls, const void* fw, void* xb, int T, int D, float eps,
                              int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  return dispatch(f32, D % 8 == 0, [&](auto ty, auto v) {
    using E = decltype(ty);
    return static_cast<int>(launch_pdl(output_norm_kernel<E, decltype(v)::value>, dim3(T), dim3(kRow), 0, s, x, reinterpret_cast<const E*>(y),
                                       reinterpret_cast<const E*>(nw), reinterpret_cast<const E*>(ls), reinterpret_cast<const E*>(fw),
                                       reinterpret_cast<E*>(xb), D, eps));
  });
}

extern "C" int mb_clamped_glu(const void* in, void* out, long long T, int F, float limit, float alpha, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  return dispatch(f32, F % 8 == 0, [&](auto ty, auto v) {
    using E = decltype(ty);
    constexpr int V = decltype(v)::value;
    const long long n = T * (F / V);
    const long long blocks = (n + 255) / 256;
    return static_cast<int>(launch_pdl(clamped_glu_kernel<E, V>, dim3(static_cast<unsigned>(blocks < 148 * 16 ? blocks : 148 * 16)), dim3(256), 0,
                                       s, reinterpret_cast<const E*>(in), reinterpret_cast<E*>(out), n, F, limit, alpha));
  });
}

extern "C" int mb_gated_norm(const void* o, const void* w, const void* gate, long long gate_ld, void* out, int T, int C, float eps, int f32,
                             cudaStream_t s) {
  if (T <= 0) return 0;
  const bool vec = C % 8 == 0 && gate_ld % 8 == 0 && reinterpret_cast<uintptr_t>(gate) % 16 == 0;
  return dispatch(f32, vec, [&](auto ty, auto v) {
    using E = decltype(ty);
    return static_cast<int>(launch_pdl(gated_norm_kernel<E, decltype(v)::value>, dim3(T), dim3(kRow), 0, s, reinterpret_cast<const E*>(o),
                                       reinterpret_cast<const E*>(w), reinterpret_cast<const E*>(gate), gate_ld, reinterpret_cast<E*>(out), C,
                                       eps));
  });
}
