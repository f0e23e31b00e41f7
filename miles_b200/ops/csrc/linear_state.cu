// Linear attention with a constant decay per head: S_t = λ S_{t−1} + k_t v_tᵀ, o_t = S_tᵀ q_t, with q, k, v = silu(projections).
// S is fp32, [slots, H, dk, dv], one slot per sequence; a sequence whose first token of the batch is at position 0 starts from zero.
//
//   linear_state_seq_kernel    any number of tokens per sequence, one after another (any sizes, bf16 or float)
//   linear_state_step_kernel   one token per sequence (decode): streams the state once, 16 bytes per thread and access
#include "mixers.cuh"

namespace mb {
namespace mx {

static constexpr int kTB = 16;      // tokens staged at a time
static constexpr int kCols = 32;    // state columns (of dv) per CTA

// grid (column slices, heads, sequences), 128 threads: lane = column, warp w owns the rows d ≡ w (mod 4) of the slice
template <typename T>
__global__ void __launch_bounds__(128) linear_state_seq_kernel(const T* __restrict__ proj, long long ld, const float* __restrict__ decay,
                                                               float* __restrict__ state, const int* __restrict__ slots,
                                                               const int* __restrict__ cu_q, const int* __restrict__ positions,
                                                               T* __restrict__ out, int H, int dk, int dv) {
  extern __shared__ __align__(16) float sm[];
  float* S = sm;                         // [dk][kCols]
  float* sq = S + dk * kCols;            // [kTB][dk]
  float* sk = sq + kTB * dk;             // [kTB][dk]
  float* sv = sk + kTB * dk;             // [kTB][kCols]
  float* part = sv + kTB * kCols;        // [kTB][4][kCols]
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kCols;
  const int t0 = cu_q != nullptr ? cu_q[b] : b, t1 = cu_q != nullptr ? cu_q[b + 1] : b + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col = c0 + lane;
  const long long ldo = static_cast<long long>(H) * dv;
  const int slot = slots[b];
  if (t1 <= t0) return;
  if (slot < 0) {                        // padding row of a decode batch
    for (int t = t0 + warp; t < t1; t += 4)
      if (col < dv) out[t * ldo + h * dv + col] = from_f<T>(0.f);
    return;
  }
  float* st = state + (static_cast<long long>(slot) * H + h) * dk * dv;
  const bool fresh = positions[t0] == 0;
  for (int d = warp; d < dk; d += 4) S[d * kCols + lane] = (!fresh && col < dv) ? st[static_cast<long long>(d) * dv + col] : 0.f;
  const float lam = decay[h];
  const T* pq = proj + h * dk;
  const T* pk = proj + static_cast<long long>(H) * dk + h * dk;
  const T* pv = proj + 2ll * H * dk + h * dv;
  for (int tb = t0; tb < t1; tb += kTB) {
    const int n = min(kTB, t1 - tb);
    __syncthreads();
    for (int i = threadIdx.x; i < n * dk; i += 128) {
      const int t = i / dk, d = i - t * dk;
      sq[i] = silu_t<T>(to_f(pq[(tb + t) * ld + d]));
      sk[i] = silu_t<T>(to_f(pk[(tb + t) * ld + d]));
    }
    for (int i = threadIdx.x; i < n * kCols; i += 128) {
      const int t = i / kCols, c = i - t * kCols;
      sv[i] = c0 + c < dv ? silu_t<T>(to_f(pv[(tb + t) * ld + c0 + c])) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float v = sv[t * kCols + lane];
      float o = 0.f;
      for (int d = warp; d < dk; d += 4) {
        const float s = fmaf(lam, S[d * kCols + lane], sk[t * dk + d] * v);
        S[d * kCols + lane] = s;
        o = fmaf(s, sq[t * dk + d], o);
      }
      part[(t * 4 + warp) * kCols + lane] = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * kCols; i += 128) {
      const int t = i / kCols, c = i - t * kCols;
      const float* p = part + t * 4 * kCols + c;
      if (c0 + c < dv) out[(tb + t) * ldo + h * dv + c0 + c] = from_f<T>((p[0] + p[kCols]) + (p[2 * kCols] + p[3 * kCols]));
    }
  }
  for (int d = warp; d < dk; d += 4)
    if (col < dv) st[static_cast<long long>(d) * dv + col] = S[d * kCols + lane];
}

// grid (128-column slices, heads, rows), 256 threads: lane = 4 columns, warp w owns the rows d ≡ w (mod 8).  dv % 4 == 0.
template <typename T>
__global__ void __launch_bounds__(256) linear_state_step_kernel(const T* __restrict__ proj, long long ld, const float* __restrict__ decay,
                                                                float* __restrict__ state, const int* __restrict__ slots,
                                                                const int* __restrict__ positions, T* __restrict__ out, int H, int dk,
                                                                int dv) {
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                 // [dk]
  float* sk = sq + dk;            // [dk]
  float* red = sk + dk;           // [8][128], moved up to a 16-byte boundary
  red = reinterpret_cast<float*>((reinterpret_cast<uintptr_t>(red) + 15) & ~static_cast<uintptr_t>(15));
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col = blockIdx.x * 128 + lane * 4;
  const bool on = col < dv;
  const long long ldo = static_cast<long long>(H) * dv;
  const int slot = slots[b];
  if (slot < 0) {
    if (warp == 0 && on)
      for (int j = 0; j < 4; ++j) out[b * ldo + h * dv + col + j] = from_f<T>(0.f);
    return;
  }
  float* st = state + (static_cast<long long>(slot) * H + h) * dk * dv;
  const bool fresh = positions[b] == 0;
  const T* p = proj + b * ld;
  // the state is on its way while the projections of this token are read and activated
  constexpr int U = 16;
  float4 s[U];
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int d = warp + u * 8;
    s[u] = (on && !fresh && d < dk) ? *reinterpret_cast<const float4*>(st + static_cast<long long>(d) * dv + col) : make_float4(0, 0, 0, 0);
  }
  for (int d = threadIdx.x; d < dk; d += 256) {
    sq[d] = silu_t<T>(to_f(p[h * dk + d]));
    sk[d] = silu_t<T>(to_f(p[static_cast<long long>(H) * dk + h * dk + d]));
  }
  float v[4] = {0.f, 0.f, 0.f, 0.f};
  if (on)
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = silu_t<T>(to_f(p[2ll * H * dk + h * dv + col + j]));
  const float lam = decay[h];
  __syncthreads();
  float o[4] = {0.f, 0.f, 0.f, 0.f};
  for (int d0 = 0; d0 < dk; d0 += U * 8) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int d = d0 + warp + u * 8;
      if (d0 > 0 && on && !fresh && d < dk) s[u] = *reinterpret_cast<const float4*>(st + static_cast<long long>(d) * dv + col);
      if (d < dk) {
        const float k = sk[d], q = sq[d];
        s[u].x = fmaf(lam, s[u].x, k * v[0]);
        s[u].y = fmaf(lam, s[u].y, k * v[1]);
        s[u].z = fmaf(lam, s[u].z, k * v[2]);
        s[u].w = fmaf(lam, s[u].w, k * v[3]);
        o[0] = fmaf(s[u].x, q, o[0]);
        o[1] = fmaf(s[u].y, q, o[1]);
        o[2] = fmaf(s[u].z, q, o[2]);
        o[3] = fmaf(s[u].w, q, o[3]);
        if (on) *reinterpret_cast<float4*>(st + static_cast<long long>(d) * dv + col) = s[u];
      }
      if (fresh) s[u] = make_float4(0, 0, 0, 0);
    }
  }
  *reinterpret_cast<float4*>(red + warp * 128 + lane * 4) = make_float4(o[0], o[1], o[2], o[3]);
  __syncthreads();
  if (threadIdx.x < 128) {
    const int c = blockIdx.x * 128 + threadIdx.x;
    float r = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) r += red[w * 128 + threadIdx.x];
    if (c < dv) out[b * ldo + h * dv + c] = from_f<T>(r);
  }
}

template <typename T>
static int run(const T* proj, long long ld, const float* decay, float* state, const int* slots, const int* cu_q, const int* positions, T* out,
               int B, int H, int dk, int dv, cudaStream_t s) {
  if (cu_q == nullptr && dv % 4 == 0) {
    const size_t bytes = (2 * dk + 8 + 8 * 128) * sizeof(float);
    if (bytes > 48 * 1024) return -3;
    return static_cast<int>(launch_pdl(linear_state_step_kernel<T>, dim3((dv + 127) / 128, H, B), dim3(256), bytes, s, proj, ld, decay, state,
                                       slots, positions, out, H, dk, dv));
  }
  const size_t bytes = (static_cast<size_t>(dk) * kCols + 2 * kTB * dk + kTB * kCols + kTB * 4 * kCols) * sizeof(float);
  if (bytes > 200 * 1024) return -3;
  static bool once = false;
  if (!once) {
    const cudaError_t e = cudaFuncSetAttribute(linear_state_seq_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    once = true;
  }
  return static_cast<int>(launch_pdl(linear_state_seq_kernel<T>, dim3((dv + kCols - 1) / kCols, H, B), dim3(128), bytes, s, proj, ld, decay, state,
                                     slots, cu_q, positions, out, H, dk, dv));
}

}  // namespace mx
}  // namespace mb

using namespace mb;
using namespace mb::mx;

extern "C" int mb_linear_state(const void* proj, long long ld, const float* decay, float* state, const int* state_slots, const int* cu_q,
                               const int* positions, void* out, int B, int H, int dk, int dv, int f32, cudaStream_t s) {
  if (B <= 0) return 0;
  if (f32)
    return run(reinterpret_cast<const float*>(proj), ld, decay, state, state_slots, cu_q, positions, reinterpret_cast<float*>(out), B, H, dk, dv, s);
  return run(reinterpret_cast<const bf16*>(proj), ld, decay, state, state_slots, cu_q, positions, reinterpret_cast<bf16*>(out), B, H, dk, dv, s);
}
