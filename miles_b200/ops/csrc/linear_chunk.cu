// Prefill of linear attention with a constant decay per head (see linear_state.cu) in chunks of 64 tokens on tensor cores.
//
// Inside a chunk, with i, j the places of two of its tokens and S the state before it,
//     o_i = λ^(i+1) Sᵀ q_i + Σ_{j ≤ i} λ^(i−j) (q_i·k_j) v_j          S ← λ^n S + Σ_j λ^(n−1−j) k_j v_jᵀ
// The state stays in fp32 registers; where it, the decayed scores and the decayed keys enter a product they are split into two
// bf16 parts (hi + lo, 16 bits of mantissa).  q, k and v are bf16 after their activation.
//
// Long prompts are cut into segments so that one sequence fills the GPU:
//   1. linear_chunk_kernel<false>   per (segment, head): the state its tokens add, from zero
//   2. linear_scan_kernel           per (sequence, head, element): state at the start of every segment
//   3. linear_chunk_kernel<true>    per (segment, head): outputs; a sequence's last segment writes its state slot
// With one segment per sequence only the third runs, straight from and to the state slots.
#include "mixers.cuh"

namespace mb {
namespace lc {

using mx::bf16;
static constexpr int C = 64, P = 136, PP = C + 8, kThreads = 512;      // tokens per chunk, shared row lengths
static constexpr int kTile = C * P;                                    // elements of a q / k / v tile (≤ 128 wide)
static constexpr size_t kSmemSums = 6 * kTile * 2 + (C + 1) * 4 + 12;      // without state and scores: two CTAs per SM
static constexpr size_t kSmem = (6 * kTile + 2 * 128 * P + 2 * C * PP) * 2 + (C + 1) * 4 + 12;

__device__ __forceinline__ uint32_t s_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void cp16(void* dst, const void* src, bool valid) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s_addr(dst)), "l"(src), "r"(sz) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float lo16(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float hi16(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}
// (a, b) = hi + lo, two bf16 pairs
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack2(a, b);
  lo = pack2(a - lo16(hi), b - hi16(hi));
}
// λ^m by repeated squaring: exact for λ = 0 and 1, a few ulp otherwise
__device__ __forceinline__ float ipow(float lam, int m) {
  float r = 1.f;
  for (; m > 0; m >>= 1, lam *= lam)
    if (m & 1) r *= lam;
  return r;
}

// silu of two values with one reciprocal: 1/a = b · 1/(ab).  Arguments below −40 count as −40 in the exponential (the result is
// zero to 15 digits either way), which keeps the product finite.
__device__ __forceinline__ void silu2(float& x, float& y) {
  const float a = 1.f + __expf(fminf(-x, 40.f)), b = 1.f + __expf(fminf(-y, 40.f));
  const float r = __fdividef(1.f, a * b);
  x *= r * b;
  y *= r * a;
}

struct Args {
  const bf16* proj;          // [T, ld]: q [H, dk], k [H, dk], v [H, dv] side by side
  long long ld;
  const float* decay;        // [H]
  float* state;              // [slots, H, dk, dv]
  const int* slots;          // per sequence
  const int* positions;      // per token
  const int* segs;           // [n_seg][4]: sequence, first token, end, 1 if the sequence's last segment
  float* seg_state;          // [n_seg, H, dk, dv]; null: one segment per sequence
  bf16* out;                 // [T, H·dv]
  int H, dk, dv;
};

// grid (heads, segments), 512 threads.  KD, VD: dk and dv when known at compile time, 0 otherwise.
template <bool OUT, int KD, int VD>
__global__ void __launch_bounds__(kThreads, OUT ? 1 : 2) linear_chunk_kernel(Args a) {
  extern __shared__ __align__(128) uint8_t smem[];
  bf16* tile = reinterpret_cast<bf16*>(smem);        // [2][q | k | v][C][P]
  bf16* s_hi = tile + 6 * kTile;                     // [128][P]
  bf16* s_lo = s_hi + 128 * P;
  bf16* p_hi = s_lo + 128 * P;                       // [C][PP]
  bf16* p_lo = p_hi + C * PP;
  float* pw = reinterpret_cast<float*>(OUT ? p_lo + C * PP : s_hi);   // λ^0 … λ^C
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, seg = blockIdx.y;
  const int seq = a.segs[seg * 4], t0 = a.segs[seg * 4 + 1], t1 = a.segs[seg * 4 + 2], last = a.segs[seg * 4 + 3];
  if (!OUT && last) return;                          // nobody continues from a last segment's own sum
  const int slot = a.slots[seq];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const float lam = a.decay[h];
  if (threadIdx.x <= C) pw[threadIdx.x] = ipow(lam, threadIdx.x);
  const int dk = KD ? KD : a.dk, dv = VD ? VD : a.dv, kdk = (dk + 15) / 16, kdv = (dv + 15) / 16;
  const long long HK = static_cast<long long>(a.H) * dk;
  const bf16* src[3] = {a.proj + h * dk, a.proj + HK + h * dk, a.proj + 2 * HK + h * dv};
  // columns [width, 16·⌈width/16⌉) of the tiles are zero for good
  for (int i = threadIdx.x; i < 6 * C; i += kThreads) {
    const int which = (i / C) % 3, w = which == 2 ? dv : dk;
    bf16* row = tile + i * P;
    for (int c = w; c < (w + 15) / 16 * 16; ++c) row[c] = __float2bfloat16(0.f);
  }
  // pieces of 8 elements: a thread activates the pieces it copied itself
  const int pk = dk / 8, pv = dv / 8, n_piece = OUT ? C * (2 * pk + pv) : C * (pk + pv);
  auto each = [&](auto&& fn) {
    for (int i = threadIdx.x; i < n_piece; i += kThreads) {
      int which, j = i, w = pk;
      if (OUT && j < C * pk) which = 0;
      else {
        if (OUT) j -= C * pk;
        if (j < C * pk) which = 1;
        else { j -= C * pk; which = 2; w = pv; }
      }
      fn(which, j / w, (j % w) * 8);
    }
  };
  auto load = [&](int c, int st) {
    const int tb = t0 + c * C;
    each([&](int which, int r, int col) {
      const bool ok = tb + r < t1;
      cp16(tile + (st * 3 + which) * kTile + r * P + col, src[which] + static_cast<long long>(ok ? tb + r : t0) * a.ld + col, ok);
    });
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(0, 0);
  // state: warp = (16 rows rt of dk, 64-column half ch of dv)
  const int rt = warp >> 1, ch = warp & 1;
  float s[8][4];
  const long long sz = static_cast<long long>(dk) * dv;
  float* slot_p = a.state + (static_cast<long long>(slot) * a.H + h) * sz;
  float* seg_p = a.seg_state != nullptr ? a.seg_state + (static_cast<long long>(seg) * a.H + h) * sz : nullptr;
  const float* init = !OUT ? nullptr : seg_p != nullptr ? seg_p : a.positions[t0] > 0 ? slot_p : nullptr;
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = rt * 16 + half * 8 + g, c = ch * 64 + n * 8 + t4 * 2;
      float2 v = make_float2(0.f, 0.f);
      if (init != nullptr && r < dk && c < dv) v = *reinterpret_cast<const float2*>(init + static_cast<long long>(r) * dv + c);
      s[n][half * 2] = v.x;
      s[n][half * 2 + 1] = v.y;
    }
  const int mt = warp >> 2, cq = warp & 3;           // scores and outputs: warp = (16 tokens, quarter of the keys / of dv)
  const int chunks = (t1 - t0 + C - 1) / C;
  auto activate = [&](int st) {
    each([&](int which, int r, int col) {
      bf16* p = tile + (st * 3 + which) * kTile + r * P + col;
      float f[8];
      mx::load_n<8>(p, f);
#pragma unroll
      for (int j = 0; j < 8; j += 2) silu2(f[j], f[j + 1]);
      mx::store_n<8>(p, f);
    });
  };
  auto publish_state = [&]() {
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = rt * 16 + half * 8 + g, c = ch * 64 + n * 8 + t4 * 2;
        uint32_t hi, lo;
        split2(s[n][half * 2], s[n][half * 2 + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(s_hi + r * P + c) = hi;
        *reinterpret_cast<uint32_t*>(s_lo + r * P + c) = lo;
      }
  };
  // Two barriers per chunk: [scores and Sᵀq] | [P·v, state update, state published, next chunk activated].  The activation of one
  // warp overlaps the products of another; the copy of chunk i + 2 runs from the first barrier to the end of the second phase.
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  activate(0);
  if (OUT) publish_state();
  for (int ci = 0; ci < chunks; ++ci) {
    const int st = ci & 1, n_tok = min(C, t1 - t0 - ci * C);
    bf16* tq = tile + st * 3 * kTile;
    bf16* tk = tq + kTile;
    bf16* tv = tk + kTile;
    __syncthreads();
    if (ci + 1 < chunks) load(ci + 1, st ^ 1);
    float o[4][4];
#pragma unroll
    for (int n = 0; n < 4; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    if (OUT) {
      float sc[2][4] = {};
      const bool seen = cq <= mt;                    // some key of the quarter is not after every token of the tile
      for (int ks = 0; ks < kdk; ++ks) {
        uint32_t aq[4], b[4];
        ldsm4(s_addr(tq + (mt * 16 + (lane & 15)) * P + ks * 16 + (lane >> 4) * 8), aq);
        if (seen) {
          ldsm4(s_addr(tk + (cq * 16 + (lane & 7) + ((lane >> 4) << 3)) * P + ks * 16 + ((lane >> 3) & 1) * 8), b);
          mma(sc[0], aq, b[0], b[1]);
          mma(sc[1], aq, b[2], b[3]);
        }
        const int srow = ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          if (cq * 2 + n < kdv) {
            const int off = srow * P + (cq * 2 + n) * 16 + (lane >> 4) * 8;
            ldsm4t(s_addr(s_hi + off), b);
            mma(o[2 * n], aq, b[0], b[1]);
            mma(o[2 * n + 1], aq, b[2], b[3]);
            ldsm4t(s_addr(s_lo + off), b);
            mma(o[2 * n], aq, b[0], b[1]);
            mma(o[2 * n + 1], aq, b[2], b[3]);
          }
        }
      }
      const float d0 = pw[mt * 16 + g + 1], d1 = pw[mt * 16 + g + 9];
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        o[n][0] *= d0; o[n][1] *= d0;
        o[n][2] *= d1; o[n][3] *= d1;
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = mt * 16 + half * 8 + g, j = cq * 16 + n * 8 + t4 * 2;
          uint32_t hi, lo;
          split2(j <= i ? sc[n][half * 2] * pw[i - j] : 0.f, j + 1 <= i ? sc[n][half * 2 + 1] * pw[i - j - 1] : 0.f, hi, lo);
          *reinterpret_cast<uint32_t*>(p_hi + i * PP + j) = hi;
          *reinterpret_cast<uint32_t*>(p_lo + i * PP + j) = lo;
        }
      __syncthreads();
      for (int ks = 0; ks <= mt; ++ks) {
        uint32_t ph[4], pl[4], b[4];
        ldsm4(s_addr(p_hi + (mt * 16 + (lane & 15)) * PP + ks * 16 + (lane >> 4) * 8), ph);
        ldsm4(s_addr(p_lo + (mt * 16 + (lane & 15)) * PP + ks * 16 + (lane >> 4) * 8), pl);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          if (cq * 2 + n < kdv) {
            ldsm4t(s_addr(tv + (ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * P + (cq * 2 + n) * 16 + (lane >> 4) * 8), b);
            mma(o[2 * n], ph, b[0], b[1]);
            mma(o[2 * n + 1], ph, b[2], b[3]);
            mma(o[2 * n], pl, b[0], b[1]);
            mma(o[2 * n + 1], pl, b[2], b[3]);
          }
        }
      }
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = mt * 16 + half * 8 + g, c = cq * 32 + n * 8 + t4 * 2;
          if (i < n_tok && c < dv)
            *reinterpret_cast<uint32_t*>(a.out + static_cast<long long>(t0 + ci * C + i) * a.H * dv + h * dv + c) = pack2(o[n][half * 2], o[n][half * 2 + 1]);
        }
    }
    // S ← λ^n S + (λ^(n−1−j) k_j)ᵀ v: the keys are decayed and split in registers
    if (rt < kdk) {
      const float dn = pw[n_tok];
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        s[n][0] *= dn; s[n][1] *= dn; s[n][2] *= dn; s[n][3] *= dn;
      }
#pragma unroll
      for (int ks = 0; ks < C / 16; ++ks) {
        uint32_t kt[4], kh[4], kl[4], b[4];
        ldsm4t(s_addr(tk + (ks * 16 + ((lane >> 4) << 3) + (lane & 7)) * P + rt * 16 + ((lane >> 3) & 1) * 8), kt);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int tok = ks * 16 + (j >> 1) * 8 + t4 * 2;
          const float f0 = tok < n_tok ? pw[n_tok - 1 - tok] : 0.f, f1 = tok + 1 < n_tok ? pw[n_tok - 2 - tok] : 0.f;
          split2(lo16(kt[j]) * f0, hi16(kt[j]) * f1, kh[j], kl[j]);
        }
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          if (ch * 4 + n < kdv) {
            ldsm4t(s_addr(tv + (ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * P + (ch * 4 + n) * 16 + (lane >> 4) * 8), b);
            mma(s[2 * n], kh, b[0], b[1]);
            mma(s[2 * n + 1], kh, b[2], b[3]);
            mma(s[2 * n], kl, b[0], b[1]);
            mma(s[2 * n + 1], kl, b[2], b[3]);
          }
        }
      }
    }
    if (ci + 1 < chunks) {
      if (OUT) publish_state();
      asm volatile("cp.async.wait_group 0;" ::: "memory");
      activate(st ^ 1);
    }
  }
  float* dst = OUT ? (last ? slot_p : nullptr) : seg_p;
  if (dst == nullptr || (OUT && slot < 0)) return;
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = rt * 16 + half * 8 + g, c = ch * 64 + n * 8 + t4 * 2;
      if (r < dk && c < dv) *reinterpret_cast<float2*>(dst + static_cast<long long>(r) * dv + c) = make_float2(s[n][half * 2], s[n][half * 2 + 1]);
    }
}

// grid (elements / 1024, heads, sequences): seg_state[i] ← state before segment i (4 elements per thread)
__global__ void __launch_bounds__(256) linear_scan_kernel(const float* __restrict__ state, const int* __restrict__ slots,
                                                          const int* __restrict__ positions, const float* __restrict__ decay,
                                                          const int* __restrict__ segs, const int* __restrict__ seq_segs,
                                                          float* seg_state, int H, int sz) {
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.y, b = blockIdx.z;
  const int e = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (e >= sz) return;
  const int s0 = seq_segs[b], s1 = seq_segs[b + 1];
  const float lam = decay[h];
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  if (positions[segs[s0 * 4 + 1]] > 0) S = *reinterpret_cast<const float4*>(state + (static_cast<long long>(slots[b]) * H + h) * sz + e);
  constexpr int U = 4;
  for (int i0 = s0; i0 < s1; i0 += U) {
    float4 add[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (i0 + u < s1 - 1) add[u] = *reinterpret_cast<const float4*>(seg_state + (static_cast<long long>(i0 + u) * H + h) * sz + e);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u;
      if (i >= s1) break;
      *reinterpret_cast<float4*>(seg_state + (static_cast<long long>(i) * H + h) * sz + e) = S;
      if (i < s1 - 1) {
        const float d = ipow(lam, segs[i * 4 + 2] - segs[i * 4 + 1]);
        S.x = fmaf(d, S.x, add[u].x);
        S.y = fmaf(d, S.y, add[u].y);
        S.z = fmaf(d, S.z, add[u].z);
        S.w = fmaf(d, S.w, add[u].w);
      }
    }
  }
}

}  // namespace lc
}  // namespace mb

using namespace mb;
using namespace mb::lc;

// bf16; dk, dv multiples of 8, ≤ 128; rows of proj 16-byte aligned.  segs [n_seg][4] and seq_segs [n_seq + 1] describe the first n_seq
// sequences of the batch; seg_state [n_seg, H, dk, dv] scratch, null when every sequence is one segment.
extern "C" int mb_linear_chunk(const void* proj, long long ld, const float* decay, float* state, const int* slots, const int* positions,
                               const int* segs, const int* seq_segs, float* seg_state, void* out, int n_seq, int n_seg, int H, int dk, int dv,
                               cudaStream_t s) {
  if (n_seg <= 0) return 0;
  if (dk % 8 || dv % 8 || dk > 128 || dv > 128 || ld % 8 || n_seg > 65535) return -3;
  const bool big = dk == 128 && dv == 128;
  auto outputs = big ? linear_chunk_kernel<true, 128, 128> : linear_chunk_kernel<true, 0, 0>;
  auto sums = big ? linear_chunk_kernel<false, 128, 128> : linear_chunk_kernel<false, 0, 0>;
  static bool once[2] = {false, false};
  if (!once[big]) {
    cudaError_t e = cudaFuncSetAttribute(outputs, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kSmem));
    if (e == cudaSuccess) e = cudaFuncSetAttribute(sums, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kSmemSums));
    if (e != cudaSuccess) return static_cast<int>(e);
    once[big] = true;
  }
  Args a{reinterpret_cast<const bf16*>(proj), ld, decay, state, slots, positions, segs, seg_state, reinterpret_cast<bf16*>(out), H, dk, dv};
  cudaError_t e = cudaSuccess;
  if (seg_state != nullptr) {
    e = launch_pdl(sums, dim3(H, n_seg), dim3(kThreads), kSmemSums, s, a);
    if (e == cudaSuccess)
      e = launch_pdl(linear_scan_kernel, dim3((dk * dv + 1023) / 1024, H, n_seq), dim3(256), 0, s, static_cast<const float*>(state), slots,
                     positions, decay, segs, seq_segs, seg_state, H, dk * dv);
  }
  if (e == cudaSuccess) e = launch_pdl(outputs, dim3(H, n_seg), dim3(kThreads), kSmem, s, a);
  return static_cast<int>(e);
}
