// Routed experts (clamped gated ones, or ungated ones with the square of relu) of any size (bf16 or float) without sorting: one row of activations per (token, choice), then one output row
// per token.  The form of 32-bit runs and of sizes the tensor-core kernels do not take; every weight row is read by one warp.
#include "mixers.cuh"

namespace mb {
namespace mx {

static constexpr int kExp = 256;

// act[pair, f] = clamped_glu(W13[e][f]·x, W13[e][F + f]·x), or with alpha = 0 relu(W13[e][f]·x)² of [E, F, H] experts.  grid (pairs, feature blocks of 8 warps)
template <typename T>
__global__ void __launch_bounds__(kExp) experts_up_kernel(const T* __restrict__ x, const T* __restrict__ w13, const int* __restrict__ index,
                                                          T* __restrict__ act, int k, int E, int H, int F, float limit, float alpha,
                                                          float shift) {
  extern __shared__ float xs[];
  pdl_trigger();
  pdl_wait();
  const long long pair = blockIdx.x, t = pair / k;
  const int e = index[pair];
  if (e < 0 || e >= E) return;                 // never read by the second kernel
  for (int i = threadIdx.x; i < H; i += kExp) xs[i] = to_f(x[t * H + i]);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int f = blockIdx.y * (kExp / 32) + warp; f < F; f += gridDim.y * (kExp / 32)) {
    const bool gated = alpha != 0.f;
    const T* g = w13 + (static_cast<long long>(e) * (gated ? 2 : 1) * F + f) * H;
    const T* u = gated ? g + static_cast<long long>(F) * H : g;
    float a = 0.f, b = 0.f;
    for (int i = lane; i < H; i += 32) {
      a = fmaf(to_f(g[i]), xs[i], a);
      if (gated) b = fmaf(to_f(u[i]), xs[i], b);
    }
    a = warp_sum(a);
    b = warp_sum(b);
    if (lane == 0) act[pair * F + f] = from_f<T>(gated ? clamped_glu_t<T>(a, b, limit, alpha, shift) : relu_square(a));
  }
}

// out[t, h] = Σ_j weights[t, j] · (W2[e][h]·act[t·k + j])
template <typename T>
__global__ void __launch_bounds__(kExp) experts_down_kernel(const T* __restrict__ act, const T* __restrict__ w2, const int* __restrict__ index,
                                                            const float* __restrict__ weights, T* __restrict__ out, int k, int E, int H, int F) {
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int h = blockIdx.y * (kExp / 32) + warp; h < H; h += gridDim.y * (kExp / 32)) {
    float s = 0.f;
    for (int j = 0; j < k; ++j) {
      const int e = index[t * k + j];
      if (e < 0 || e >= E) continue;
      const T* w = w2 + (static_cast<long long>(e) * H + h) * F;
      const T* a = act + (t * k + j) * F;
      float d = 0.f;
      for (int f = lane; f < F; f += 32) d = fmaf(to_f(w[f]), to_f(a[f]), d);
      s = fmaf(weights[t * k + j], d, s);
    }
    s = warp_sum(s);
    if (lane == 0) out[t * H + h] = from_f<T>(s);
  }
}

}  // namespace mx
}  // namespace mb

using namespace mb;
using namespace mb::mx;

// x [T, H], w13 [E, 2F, H] (alpha 0: [E, F, H]), w2 [E, H, F], index / weights [T, k]; act [T·k, F] scratch, out [T, H]
extern "C" int mb_experts_any(const void* x, const void* w13, const void* w2, const int* index, const float* weights, void* act, void* out, int T,
                              int k, int E, int H, int F, float limit, float alpha, float shift, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  if (H > 12288 || k <= 0) return -3;
  auto run = [&](auto ty) {
    using P = decltype(ty);
    const int fb = (F + 7) / 8 < 64 ? (F + 7) / 8 : 64, hb = (H + 7) / 8 < 64 ? (H + 7) / 8 : 64;
    cudaError_t e = launch_pdl(experts_up_kernel<P>, dim3(static_cast<unsigned>(T) * k, fb), dim3(kExp), H * sizeof(float), s,
                               reinterpret_cast<const P*>(x), reinterpret_cast<const P*>(w13), index, reinterpret_cast<P*>(act), k, E, H, F, limit,
                               alpha, shift);
    if (e == cudaSuccess)
      e = launch_pdl(experts_down_kernel<P>, dim3(T, hb), dim3(kExp), 0, s, reinterpret_cast<const P*>(act), reinterpret_cast<const P*>(w2), index,
                     weights, reinterpret_cast<P*>(out), k, E, H, F);
    return static_cast<int>(e);
  };
  return f32 ? run(float{}) : run(bf16{});
}
