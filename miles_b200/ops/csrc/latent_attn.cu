// Latent attention over a paged cache of latents (any sizes, bf16 or float): rotation and caching of the new tokens' latents, per-head
// projections.  Attention in the absorbed form — the query carries the key up-projection, so keys are the cached rows
// themselves and the value up-projection follows on the attended latent — is paged_attend.cu for any size.
//
// A cached row is [latent (rank) | 0 … rank_p | rotated key part (rot) | 0 … pitch); rank_p and pitch are multiples of 16.
// An absorbed query has the same layout per head, so a score is one dot product over a row.
#include "mixers.cuh"

namespace mb {
namespace mx {

// Two CTAs per token: one rotates the rotated part of every query head (interleaved pairs, angles in double precision, so that a
// position of any size costs no accuracy); the other RMS-norms the new latent, rotates the shared key part and writes the cache row.
// Tokens before `t_long` get a full query [H][q_width] = [unrotated | 0 … q_nope | rotated | 0 … q_width) for the expanded
// form; later ones the rotated part and the padding of an absorbed query [H][pitch] (head_linear fills [0, rank)).
// VEC: rows and head parts start on 16-byte boundaries and are whole 16-byte pieces.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) latent_prep_kernel(const T* __restrict__ q_in, long long q_ld, const T* __restrict__ kv_in, long long kv_ld,
                                                          const int* __restrict__ positions,
                                                          const long long* __restrict__ slots, const double* __restrict__ freq,
                                                          float magnitude, const T* __restrict__ kv_norm, float eps,
                                                          T* __restrict__ cache, T* __restrict__ q_abs, T* __restrict__ q_full, int t_long,
                                                          int q_nope, int q_width, MbLatent L) {
  extern __shared__ float cs[];          // [rot/2] cosines, [rot/2] sines
  __shared__ float sh[8];
  constexpr int V = VEC ? 16 / static_cast<int>(sizeof(T)) : 2;      // values per piece (a piece is whole pairs)
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const int half = L.rot / 2, dq = L.dim + L.rot;
  const T* p = q_in + t * q_ld;
  rotary_table<T, 256>(cs, positions[t], freq, half, magnitude);
  auto rotate = [&](float (&f)[V], int k) {      // V values, the first one the even half of pair k
#pragma unroll
    for (int j = 0; j < V; j += 2) {
      const float u = f[j], v = f[j + 1], c = cs[k + j / 2], s = cs[half + k + j / 2];
      f[j] = u * c - v * s;
      f[j + 1] = v * c + u * s;
    }
  };
  if (blockIdx.y == 0) {
    const bool full = t < t_long;
    T* q = full ? q_full + t * static_cast<long long>(L.heads) * q_width : q_abs + (t - t_long) * static_cast<long long>(L.heads) * L.pitch;
    const int width = full ? q_width : L.pitch, rot_at = full ? q_nope : L.rank_p, filled = full ? L.dim : L.rank;
    if (full) {
      const int n = L.dim / V, rest = L.dim - n * V;
#pragma unroll 4
      for (int i = threadIdx.x; i < L.heads * n; i += 256) {
        const int h = i / n, c = (i - h * n) * V;
        float f[V];
        load_n<V>(p + h * dq + c, f);
        store_n<V>(q + h * width + c, f);
      }
      if (rest)
        for (int h = threadIdx.x; h < L.heads; h += 256) q[h * width + L.dim - 1] = p[h * dq + L.dim - 1];
    }
    __syncthreads();
    const int n = L.rot / V;
#pragma unroll 4
    for (int i = threadIdx.x; i < L.heads * n; i += 256) {
      const int h = i / n, c = (i - h * n) * V;
      float f[V];
      load_n<V>(p + h * dq + L.dim + c, f);
      rotate(f, c / 2);
      store_n<V>(q + h * width + rot_at + c, f);
    }
    const int gap = rot_at - filled, tail = width - rot_at - L.rot;
    for (int i = threadIdx.x; i < L.heads * (gap + tail); i += 256) {
      const int h = i / (gap + tail), c = i - h * (gap + tail);
      q[h * width + (c < gap ? filled + c : rot_at + L.rot + c - gap)] = from_f<T>(0.f);
    }
    return;
  }
  const long long slot = slots[t];
  if (slot < 0) return;
  const T* kv = kv_in + t * kv_ld;
  float ss = 0.f;
  for (int i = threadIdx.x; i < L.rank; i += 256) {
    const float v = to_f(kv[i]);
    ss += v * v;
  }
  const float rstd = rsqrt_exact(__fdiv_rn(block_sum<256>(ss, sh), static_cast<float>(L.rank)) + eps);      // (also orders cs)
  T* row = cache + slot * L.pitch;
  for (int i = threadIdx.x; i < L.pitch; i += 256) {
    float v = 0.f;
    if (i < L.rank) {
      v = to_f(kv[i]) * rstd * to_f(kv_norm[i]);
    } else if (i >= L.rank_p && i < L.rank_p + L.rot) {
      const int r = i - L.rank_p, k = r >> 1;
      const float a = to_f(kv[L.rank + 2 * k]), b = to_f(kv[L.rank + 2 * k + 1]);
      v = (r & 1) ? b * cs[k] + a * cs[half + k] : a * cs[k] - b * cs[half + k];
    }
    row[i] = from_f<T>(v);
  }
}

// y[t, h, n] = Σ_k x[t, h, k] · w[h](n, k); w [H, N, K] when NK, else [H, K, N].  Any sizes; one output per thread.
template <typename T, bool NK>
__global__ void __launch_bounds__(128) head_linear_kernel(const T* __restrict__ x, long long x_t, long long x_h, const T* __restrict__ w,
                                                          T* __restrict__ y, long long y_t, long long y_h, int N, int K,
                                                          const T* __restrict__ gate, long long gate_ld) {
  extern __shared__ float xs[];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.z;
  const int h = blockIdx.y, n = blockIdx.x * 128 + threadIdx.x;
  for (int k = threadIdx.x; k < K; k += 128) xs[k] = to_f(x[t * x_t + h * x_h + k]);
  __syncthreads();
  if (n >= N) return;
  const T* wh = w + static_cast<long long>(h) * N * K + (NK ? static_cast<long long>(n) * K : n);
  float s = 0.f;
  for (int k = 0; k < K; ++k) s = fmaf(xs[k], to_f(wh[NK ? k : static_cast<long long>(k) * N]), s);
  if (gate != nullptr) s *= sigmoid_t<T>(to_f(gate[t * gate_ld + h * N + n]));
  y[t * y_t + h * y_h + n] = from_f<T>(s);
}

template <typename T>
static int prep(const T* q, long long q_ld, const T* kv, long long kv_ld, const int* positions, const long long* slots, const double* freq, float magnitude,
                const T* kv_norm, float eps, T* cache, T* q_abs, T* q_full, int n, int t_long, int q_nope, int q_width, MbLatent L,
                cudaStream_t s) {
  if (L.rot > 4096 || L.rot % 2) return -3;
  const int v = 16 / static_cast<int>(sizeof(T));
  const bool vec = q_ld % v == 0 && L.dim % v == 0 && L.rot % v == 0 && q_nope % v == 0 && q_width % v == 0 && reinterpret_cast<uintptr_t>(q) % 16 == 0;
  const dim3 grid(n, kv_norm != nullptr ? 2 : 1);
  auto kern = vec ? latent_prep_kernel<T, true> : latent_prep_kernel<T, false>;
  return static_cast<int>(launch_pdl(kern, grid, dim3(256), L.rot * sizeof(float), s, q, q_ld, kv, kv_ld, positions, slots, freq, magnitude, kv_norm, eps,
                                     cache, q_abs, q_full, t_long, q_nope, q_width, L));
}

template <typename T>
static int head_linear(const T* x, long long x_t, long long x_h, const T* w, int nk, T* y, long long y_t, long long y_h, int n, int H, int N,
                       int K, const T* gate, long long gate_ld, cudaStream_t s) {
  if (K > 8192) return -3;
  for (int t0 = 0; t0 < n; t0 += 65535) {
    const dim3 grid((N + 127) / 128, H, n - t0 < 65535 ? n - t0 : 65535);
    const cudaError_t e = launch_pdl(nk ? head_linear_kernel<T, true> : head_linear_kernel<T, false>, grid, dim3(128), K * sizeof(float), s, x + t0 * x_t, x_t,
                                     x_h, w, y + t0 * y_t, y_t, y_h, N, K, gate != nullptr ? gate + t0 * gate_ld : gate, gate_ld);
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  return 0;
}

}  // namespace mx
}  // namespace mb

using namespace mb;
using namespace mb::mx;

#define MB_BY_TYPE(call)                          \
  if (f32) { using E = float; return call; }      \
  using E = bf16;                                 \
  return call

extern "C" int mb_latent_prep(const void* q, long long q_ld, const void* kv, long long kv_ld, const int* positions, const long long* slots, const double* freq,
                              float magnitude, const void* kv_norm, float eps, void* cache, void* q_abs, void* q_full, int T, int t_long,
                              int q_nope, int q_width, MbLatent L, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  MB_BY_TYPE(prep(reinterpret_cast<const E*>(q), q_ld, reinterpret_cast<const E*>(kv), kv_ld, positions, slots, freq, magnitude, reinterpret_cast<const E*>(kv_norm), eps,
                  reinterpret_cast<E*>(cache), reinterpret_cast<E*>(q_abs), reinterpret_cast<E*>(q_full), T, t_long, q_nope, q_width, L, s));
}

extern "C" int mb_head_linear(const void* x, long long x_t, long long x_h, const void* w, int w_nk, void* y, long long y_t, long long y_h,
                              int T, int H, int N, int K, const void* gate, long long gate_ld, int f32, cudaStream_t s) {
  if (T <= 0) return 0;
  MB_BY_TYPE(head_linear(reinterpret_cast<const E*>(x), x_t, x_h, reinterpret_cast<const E*>(w), w_nk, reinterpret_cast<E*>(y), y_t, y_h, T, H,
                         N, K, reinterpret_cast<const E*>(gate), gate_ld, s));
}

// the absorbed form on the any-size kernel: one "key head" whose keys are the cached rows and whose values are their latent part
extern "C" int mb_latent_attend(const void* q, const void* cache, const int* block_table, int max_blocks, int block_size,
                                const int* token_seq, const int* positions, const long long* slots, const void* sink, void* out, int T,
                                float scale, int window, MbLatent L, int f32, cudaStream_t s) {
  MbAttend a{};
  a.heads = a.group = L.heads;
  a.dk = L.pitch; a.dv = L.rank;
  a.q_head = L.pitch; a.q_row = static_cast<long long>(L.heads) * L.pitch;
  a.k_row = a.v_row = L.pitch;
  a.o_row = static_cast<long long>(L.heads) * L.rank;
  a.window = window;
  a.scale = scale;
  return mb_paged_attend(q, cache, cache, block_table, max_blocks, block_size, token_seq, positions, slots, sink, out, T, a, MbScores{}, f32, 0, s);
}
