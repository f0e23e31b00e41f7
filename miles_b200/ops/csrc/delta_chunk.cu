// Prefill of the gated delta rule with a decay per head and key channel (see delta_state.cu) in chunks of 64 tokens on tensor cores.
//
// With G_i the running sum of the log decays inside a chunk (per channel) and S the state before it, the tokens' updates u_i satisfy
//     (I + A) u = β v − (β k e^G) S        A_ij = β_i Σ_c k_ic k_jc e^(G_ic − G_jc), j < i
//     o_i = (q_i e^G_i) S + Σ_{j ≤ i} B_ij u_j        B_ij = Σ_c q_ic k_jc e^(G_ic − G_jc)
//     S ← e^G_last S + Σ_j (k_j e^(G_last − G_j)) u_jᵀ
// so a chunk is U = T β v, W = T β k e^G with T = (I + A)⁻¹, and u = U − W S.  Two kernels:
//   1. delta_prepare_kernel   per (chunk, head), all of them at once: unit vectors, decays, A, B, T, W, U, and the decayed queries and
//                             keys, written as the shared-memory images the second kernel wants
//   2. delta_scan_kernel      per (sequence, head, slice of value columns), chunk by chunk: u, outputs, state.  A warp owns 16 value
//                             columns: Sᵀ stays in its registers, as accumulator and as operand, so warps never exchange anything.
// Every factor of a product is at most 1 or belongs to a difference that is: decays count from the start (rows) or to the end (columns) of
// blocks of 16 tokens, and what lies between two blocks is a factor of its own.  Only inside a block do exponents of both signs meet; a
// block with a channel that decays by more than 2^100 is summed directly.
// All these quantities enter products as two bf16 parts (hi + lo, 16 bits of mantissa; three products of parts); sums are fp32.
#include "mixers.cuh"
#include "ptx.cuh"

namespace mb {
namespace dc {

using mx::bf16;
static constexpr int C = 64, kThreads = 512;
static constexpr int P = 136, LP = 132, AP = 68;      // shared rows: bf16 tiles (≤ 128 wide), floats per channel, floats per token
static constexpr int kTile = C * P;
static constexpr float kLog2e = 1.4426950408889634f, kFar = -100.f;
static constexpr int kUPitch = 288;                   // bytes of a row of U (64 floats and padding)

__device__ __forceinline__ void ldsm4(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void stsm4t(uint32_t a, uint32_t r0, uint32_t r1, uint32_t r2, uint32_t r3) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1,%2,%3,%4};" ::"r"(a), "r"(r0), "r"(r1), "r"(r2), "r"(r3) : "memory");
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
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
__device__ __forceinline__ void split8(const float (&f)[8], uint4& hi, uint4& lo) {
  split2(f[0], f[1], hi.x, lo.x);
  split2(f[2], f[3], hi.y, lo.y);
  split2(f[4], f[5], hi.z, lo.z);
  split2(f[6], f[7], hi.w, lo.w);
}
// the two 8-column accumulators (n, n + 1) of 16 rows as the 16×16 operand of the next product
__device__ __forceinline__ void operand(const float (&x)[4], const float (&y)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
  split2(x[0], x[1], hi[0], lo[0]);
  split2(x[2], x[3], hi[1], lo[1]);
  split2(y[0], y[1], hi[2], lo[2]);
  split2(y[2], y[3], hi[3], lo[3]);
}
__device__ __forceinline__ float e2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// log2(e) · softplus(x): log2(1 + y) with y = e^−|x|, by its series where 1 + y would round y away
__device__ __forceinline__ float softplus2(float x) {
  const float y = __expf(-fabsf(x));
  const float l = y < 0.0078125f ? kLog2e * y * fmaf(y, fmaf(y, fmaf(y, -0.25f, 0.33333334f), -0.5f), 1.f) : __log2f(1.f + y);
  return fmaf(fmaxf(x, 0.f), kLog2e, l);
}

// One (chunk, head) of scratch: W [KR rows of 64 tokens] hi, lo | q [64 rows of KR] hi, lo | B [64 rows of 64] hi, lo | k [64 rows of KR] hi, lo |
// decay of the chunk [128] floats | U [VP rows of 72 floats].  Rows of bf16 hold their 16-byte pieces at piece ^ (row mod 8).
struct Unit {
  int KR, VP;
  __host__ __device__ int half() const { return KR * 128; }
  __host__ __device__ int q() const { return 2 * half(); }
  __host__ __device__ int b() const { return 4 * half(); }
  __host__ __device__ int k() const { return 4 * half() + 16384; }
  __host__ __device__ int decay() const { return 6 * half() + 16384; }
  __host__ __device__ int u() const { return decay() + 512; }
  __host__ __device__ long long bytes() const { return u() + static_cast<long long>(VP) * kUPitch; }
};

struct Args {
  const bf16* proj;          // β in column m.beta_at
  long long ld;
  const bf16* act;           // [T, 2·G·K + H·V]: q, k, v after convolution and silu
  MbDelta m;
  const int* chunks;         // [n][4]: sequence, first token, end
  const int* parts;          // [n][4]: first chunk, chunks, sequence
  uint8_t* scratch;
  Unit unit;
  bf16* out;                 // [T, H·V]
  int* error_flag;
};

struct Shared {
  bf16 q_hi[kTile], q_lo[kTile], k_hi[kTile], k_lo[kTile], c_hi[kTile], c_lo[kTile], v[kTile];
  float L[C * LP];           // log2 of the decays, summed from the start of a token's block
  float A[C * AP];
  float D[4][128], before[4][128], after[4][128], between[7][128];
  float fq[C], fk[C], beta[C];
  int direct[4];
};

// (row block, column block) of the pairs whose columns take a factor: those with blocks between them, and the diagonal ones
__device__ __forceinline__ void pair_of(int i, int& a, int& b) {
  a = i < 3 ? (i == 0 ? 2 : 3) : i - 3;
  b = i < 3 ? (i == 2 ? 1 : 0) : i - 3;
}

// grid (heads, chunks)
__global__ void __launch_bounds__(kThreads, 1) delta_prepare_kernel(Args p) {
  extern __shared__ __align__(128) uint8_t smem[];
  Shared& s = *reinterpret_cast<Shared*>(smem);
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.x, H = p.m.H, K = p.m.K, V = p.m.V, gq = h / (H / p.m.G), CH = 2 * p.m.G * K + H * V;
  const int4 ch = reinterpret_cast<const int4*>(p.chunks)[blockIdx.y];
  const int t0 = ch.y, n_tok = ch.z - ch.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int kdk = (K + 15) / 16, kdv = (V + 15) / 16;
  uint8_t* unit = p.scratch + (static_cast<long long>(blockIdx.y) * H + h) * p.unit.bytes();
  const int KR = p.unit.KR, half = p.unit.half();

  // ---- inputs: q and k as they are (with the factors that make them unit vectors), v, log decays, β
  const float q_scale = __fdiv_rn(1.f, __fsqrt_rn(static_cast<float>(K)));
  for (int r = warp; r < C; r += kThreads / 32) {
    const int piece = lane & 15;
    const bool key = lane >= 16;
    uint4 x = make_uint4(0, 0, 0, 0);
    if (r < n_tok && piece * 8 < K) x = *reinterpret_cast<const uint4*>(p.act + static_cast<long long>(t0 + r) * CH + (key ? p.m.G * K : 0) + gq * K + piece * 8);
    const uint32_t w[4] = {x.x, x.y, x.z, x.w};
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) ss += lo16(w[i]) * lo16(w[i]) + hi16(w[i]) * hi16(w[i]);
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float f = mx::rsqrt_exact(ss + 1e-6f);
    if (piece == 0) (key ? s.fk : s.fq)[r] = key ? f : f * q_scale;
    *reinterpret_cast<uint4*>((key ? s.k_hi : s.q_hi) + r * P + piece * 8) = x;
  }
  const float rate = __expf(__bfloat162float(reinterpret_cast<const bf16*>(p.m.A_log)[h]));
  for (int i = tid; i < C * 16; i += kThreads) {
    const int r = i >> 4, c = (i & 15) * 8;
    uint4 x = make_uint4(0, 0, 0, 0);
    if (r < n_tok && c < V) x = *reinterpret_cast<const uint4*>(p.act + static_cast<long long>(t0 + r) * CH + 2 * p.m.G * K + h * V + c);
    *reinterpret_cast<uint4*>(s.v + r * P + c) = x;
    float l[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) l[j] = 0.f;
    if (r < n_tok && c < K) {
      float bias[8];
      mx::load_n<8>(reinterpret_cast<const bf16*>(p.m.raw) + (t0 + r) * p.m.raw_ld + h * K + c, l);
      mx::load_n<8>(reinterpret_cast<const bf16*>(p.m.dt_bias) + h * K + c, bias);
#pragma unroll
      for (int j = 0; j < 8; ++j) l[j] = -rate * softplus2(l[j] + bias[j]);
    }
    mx::store_n<8>(s.L + r * LP + c, l);
  }
  if (tid < C) s.beta[tid] = tid < n_tok ? mx::sigmoid_t<bf16>(__bfloat162float(p.proj[(t0 + tid) * p.ld + p.m.beta_at + h])) : 0.f;
  if (tid < 4) s.direct[tid] = 0;
  __syncthreads();
  {                                      // running sums inside the blocks: a thread per (block, channel)
    const int b = tid >> 7, c = tid & 127;
    float* x = s.L + b * 16 * LP + c;
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      sum += x[i * LP];
      x[i * LP] = sum;
    }
    s.D[b][c] = sum;
    if (sum < kFar) s.direct[b] = 1;
  }
  __syncthreads();
  if (tid < 128) {
    const float d0 = s.D[0][tid], d1 = s.D[1][tid], d2 = s.D[2][tid], d3 = s.D[3][tid];
    s.before[0][tid] = 1.f;
    s.before[1][tid] = e2(d0);
    s.before[2][tid] = e2(d0 + d1);
    s.before[3][tid] = e2(d0 + d1 + d2);
    s.after[0][tid] = e2(d1 + d2 + d3);
    s.after[1][tid] = e2(d2 + d3);
    s.after[2][tid] = e2(d3);
    s.after[3][tid] = 1.f;
    s.between[0][tid] = e2(d1);
    s.between[1][tid] = e2(d1 + d2);
    s.between[2][tid] = e2(d2);
    s.between[3][tid] = e2(fminf(-d0, -kFar));           // blocks beyond are summed directly
    s.between[4][tid] = e2(fminf(-d1, -kFar));
    s.between[5][tid] = e2(fminf(-d2, -kFar));
    s.between[6][tid] = e2(fminf(-d3, -kFar));
    reinterpret_cast<float*>(unit + p.unit.decay())[tid] = e2(d0 + d1 + d2 + d3);
  }
  // ---- q and k decayed from the start of their block, k to its end
  for (int i = tid; i < C * 16; i += kThreads) {
    const int r = i >> 4, c = (i & 15) * 8, at = r * P + c;
    float q[8], k[8], l[8], d[8], x[8];
    uint4 hi, lo;
    mx::load_n<8>(s.q_hi + at, q);
    mx::load_n<8>(s.k_hi + at, k);
    mx::load_n<8>(s.L + r * LP + c, l);
    mx::load_n<8>(s.D[r >> 4] + c, d);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      d[j] = k[j] * e2(d[j] - l[j]);
      l[j] = e2(l[j]);
      x[j] = q[j] * l[j];
    }
    split8(x, hi, lo);
    *reinterpret_cast<uint4*>(s.q_hi + at) = hi;
    *reinterpret_cast<uint4*>(s.q_lo + at) = lo;
#pragma unroll
    for (int j = 0; j < 8; ++j) x[j] = k[j] * l[j];
    split8(x, hi, lo);
    *reinterpret_cast<uint4*>(s.k_hi + at) = hi;
    *reinterpret_cast<uint4*>(s.k_lo + at) = lo;
    split8(d, hi, lo);
    *reinterpret_cast<uint4*>(s.c_hi + at) = hi;
    *reinterpret_cast<uint4*>(s.c_lo + at) = lo;
  }
  __syncthreads();
  // ---- A and B, a warp per (pair of blocks, 8 columns): 14 units with a factor on the columns, 6 of neighbouring blocks without
  for (int round = 0; round < (warp < 14 ? 1 : 3); ++round) {
    int a, b;
    const int n = warp < 14 ? warp & 1 : warp - 14;
    if (warp < 14) pair_of(warp >> 1, a, b);
    else { a = round + 1; b = round; }
    const float* fac = warp < 14 ? s.between[warp >> 1] : nullptr;
    float kk[4] = {0.f, 0.f, 0.f, 0.f}, qk[4] = {0.f, 0.f, 0.f, 0.f};
    if (a == b && s.direct[a]) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = a * 16 + g + (e >> 1) * 8, j = a * 16 + n * 8 + t4 * 2 + (e & 1);
        if (j > i || i >= n_tok) continue;
        const bf16* qi = p.act + static_cast<long long>(t0 + i) * CH + gq * K;
        const bf16* ki = qi + p.m.G * K;
        const bf16* kj = p.act + static_cast<long long>(t0 + j) * CH + p.m.G * K + gq * K;
        for (int c = 0; c < K; ++c) {
          const float x = __bfloat162float(kj[c]) * e2(s.L[i * LP + c] - s.L[j * LP + c]);
          kk[e] = fmaf(__bfloat162float(ki[c]), x, kk[e]);
          qk[e] = fmaf(__bfloat162float(qi[c]), x, qk[e]);
        }
      }
      __syncwarp();
    } else {
      const int row_a = (a * 16 + (lane & 15)) * P + (lane >> 4) * 8;
      const uint32_t b_at = smem_u32((lane < 16 ? s.c_hi : s.c_lo) + (b * 16 + n * 8 + (lane & 7)) * P + ((lane >> 3) & 1) * 8);
      for (int ks = 0; ks < kdk; ++ks) {
        uint32_t qh[4], ql[4], kh[4], kl[4], c[4];
        ldsm4(b_at + ks * 32, c);                        // hi: c[0], c[1]; lo: c[2], c[3]
        ldsm4(smem_u32(s.k_hi + row_a + ks * 16), kh);
        ldsm4(smem_u32(s.k_lo + row_a + ks * 16), kl);
        ldsm4(smem_u32(s.q_hi + row_a + ks * 16), qh);
        ldsm4(smem_u32(s.q_lo + row_a + ks * 16), ql);
        if (fac != nullptr) {
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const float2 f = *reinterpret_cast<const float2*>(fac + ks * 16 + i * 8 + t4 * 2);
            split2((lo16(c[i]) + lo16(c[2 + i])) * f.x, (hi16(c[i]) + hi16(c[2 + i])) * f.y, c[i], c[2 + i]);
          }
        }
        mma(kk, kh, c[0], c[1]);
        mma(qk, qh, c[0], c[1]);
        mma(kk, kh, c[2], c[3]);
        mma(qk, qh, c[2], c[3]);
        mma(kk, kl, c[0], c[1]);
        mma(qk, ql, c[0], c[1]);
      }
    }
#pragma unroll
    for (int e = 0; e < 4; e += 2) {
      const int i = a * 16 + g + e * 4, j = b * 16 + n * 8 + t4 * 2;
      const float f0 = s.fk[j], f1 = s.fk[j + 1], fi = s.fk[i] * s.beta[i], fo = s.fq[i];
      *reinterpret_cast<float2*>(s.A + i * AP + j) = make_float2(j < i ? kk[e] * fi * f0 : 0.f, j + 1 < i ? kk[e + 1] * fi * f1 : 0.f);
      uint32_t hi, lo;
      split2(j <= i ? qk[e] * fo * f0 : 0.f, j + 1 <= i ? qk[e + 1] * fo * f1 : 0.f, hi, lo);
      uint8_t* at = unit + p.unit.b() + i * 128 + (((j >> 3) ^ (i & 7)) << 4) + (j & 7) * 2;
      *reinterpret_cast<uint32_t*>(at) = hi;
      *reinterpret_cast<uint32_t*>(at + 8192) = lo;
    }
  }
  __syncthreads();
  if (warp < 4) {
    // ---- inverses of the diagonal blocks of I + A, over them: a lane per column
    const int c = lane & 15;
    float* blk = s.A + warp * 16 * AP + warp * 16;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float r = i == c ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) r = fmaf(-blk[i * AP + j], x[j], r);
      x[i] = r;
    }
    __syncwarp();
    if (lane < 16)
#pragma unroll
      for (int i = 0; i < 16; ++i) blk[i * AP + c] = x[i];
  } else {
    // ---- queries decayed from the chunk's start, keys to its end
    for (int i = tid - 128; i < 2 * C * 16; i += kThreads - 128) {
      const int r = (i >> 4) & (C - 1), piece = i & 15, c = piece * 8, at = r * P + c;
      const bool key = i >= C * 16;
      if (c >= kdk * 16) continue;
      float x[8], y[8];
      mx::load_n<8>((key ? s.c_hi : s.q_hi) + at, x);
      mx::load_n<8>((key ? s.c_lo : s.q_lo) + at, y);
      const float* f = (key ? s.after : s.before)[r >> 4] + c;
      const float scale = key ? s.fk[r] : s.fq[r];
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] = (x[j] + y[j]) * (f[j] * scale);
      uint4 hi, lo;
      split8(x, hi, lo);
      uint8_t* to = unit + (key ? p.unit.k() : p.unit.q()) + r * KR * 2 + ((piece ^ (r & 7)) << 4);
      *reinterpret_cast<uint4*>(to) = hi;
      *reinterpret_cast<uint4*>(to + half) = lo;
    }
  }
  __syncthreads();
  // ---- X = T·[β v | β k e^G] by blocks of tokens, transposed: a warp's 16 columns are the rows of its products
  for (int mt = warp; mt < kdv + kdk; mt += kThreads / 32) {
    const bool is_u = mt < kdv;
    const int c0 = (is_u ? mt : mt - kdv) * 16;
    uint32_t xh[4][4], xl[4][4];
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
      // rows of A (or T) are the columns of the second factor
      auto times = [&](float (&d)[2][4], const uint32_t (&yh)[4], const uint32_t (&yl)[4], int b) {
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const float* row = s.A + (a * 16 + n * 8 + g) * AP + b * 16 + t4 * 2;
          const float2 u = *reinterpret_cast<const float2*>(row), v = *reinterpret_cast<const float2*>(row + 8);
          uint32_t h0, l0, h1, l1;
          split2(u.x, u.y, h0, l0);
          split2(v.x, v.y, h1, l1);
          mma(d[n], yh, h0, h1);
          mma(d[n], yh, l0, l1);
          mma(d[n], yl, h0, h1);
        }
      };
#pragma unroll
      for (int b = 0; b < a; ++b) times(acc, xh[b], xl[b], b);
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int c = c0 + g + (e >> 1) * 8, t = a * 16 + n * 8 + t4 * 2 + (e & 1);
          float r;
          if (is_u) r = __bfloat162float(s.v[t * P + c]);
          else r = (__bfloat162float(s.k_hi[t * P + c]) + __bfloat162float(s.k_lo[t * P + c])) * (s.fk[t] * s.before[a][c]);
          acc[n][e] = fmaf(r, s.beta[t], -acc[n][e]);
        }
      uint32_t yh[4], yl[4];
      operand(acc[0], acc[1], yh, yl);
      float x[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
      times(x, yh, yl, a);
      operand(x[0], x[1], xh[a], xl[a]);
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int c = c0 + g + e * 8, t = a * 16 + n * 8 + t4 * 2;
          if (is_u) {
            *reinterpret_cast<float2*>(unit + p.unit.u() + c * kUPitch + t * 4) = make_float2(x[n][e * 2], x[n][e * 2 + 1]);
          } else {                       // −W: the second kernel adds
            uint8_t* to = unit + c * 128 + (((t >> 3) ^ (c & 7)) << 4) + (t & 7) * 2;
            *reinterpret_cast<uint32_t*>(to) = xh[a][n * 2 + e] ^ 0x80008000u;
            *reinterpret_cast<uint32_t*>(to + half) = xl[a][n * 2 + e] ^ 0x80008000u;
          }
        }
    }
  }
}

__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}

static size_t scan_bytes(const Unit& u, int warps) { return static_cast<size_t>(u.u()) + warps * (16 * kUPitch + 2048) + 64; }

// grid (slices of 16·NW value columns, heads, parts of sequences), 32·NW threads
template <int NW>
__global__ void __launch_bounds__(32 * NW, 1) delta_scan_kernel(Args p) {
  extern __shared__ __align__(128) uint8_t smem[];
  const Unit un = p.unit;
  const int KR = un.KR, half = un.half();
  uint8_t* sU = smem + un.u();
  uint8_t* stage = sU + NW * 16 * kUPitch;
  uint64_t* bars = reinterpret_cast<uint64_t*>(stage + NW * 2048);        // W and U | q and B | k and decay
  volatile int* abort_flag = reinterpret_cast<volatile int*>(bars + 3);
  const int h = blockIdx.y, H = p.m.H, K = p.m.K, V = p.m.V, kdk = (K + 15) / 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  if (tid == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(&bars[i], 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  pdl_trigger();
  pdl_wait();
  const int4 part = reinterpret_cast<const int4*>(p.parts)[blockIdx.z];
  const int first = part.x, n_chunks = part.y, slot = p.m.slots[part.z];
  const int c_cta = blockIdx.x * NW * 16, c0 = c_cta + warp * 16;
  const int u_rows = min(NW * 16, un.VP - c_cta);
  const bool active = c0 < un.VP;        // (the last slice may be narrower)
  __syncthreads();
  auto unit_of = [&](int i) { return p.scratch + (static_cast<long long>(first + i) * H + h) * un.bytes(); };
  auto load_w = [&](int i) {
    const uint8_t* src = unit_of(i);
    mbar_expect_tx(&bars[0], 2 * half + u_rows * kUPitch);
    bulk_load(smem, src, 2 * half, &bars[0]);
    bulk_load(sU, src + un.u() + c_cta * kUPitch, u_rows * kUPitch, &bars[0]);
  };
  auto load_q = [&](int i) {
    mbar_expect_tx(&bars[1], 2 * half + 16384);
    bulk_load(smem + un.q(), unit_of(i) + un.q(), 2 * half + 16384, &bars[1]);
  };
  auto load_k = [&](int i) {
    mbar_expect_tx(&bars[2], 2 * half + 512);
    bulk_load(smem + un.k(), unit_of(i) + un.k(), 2 * half + 512, &bars[2]);
  };
  if (tid == 0) {
    load_w(0);
    load_q(0);
    load_k(0);
  }
  auto wait = [&](int which, int i) {
    if (*abort_flag) return;
    if (!mbar_wait(&bars[which], i & 1)) {
      *abort_flag = 1;
      atomicExch(p.error_flag, 91);
    }
  };
  // Sᵀ: rows are the warp's value columns g and g + 8, accumulator n holds channels 8n + 2·t4 and the next
  float* st = p.m.state + (static_cast<long long>(max(slot, 0)) * H + h) * K * V;
  const int t_first = reinterpret_cast<const int4*>(p.chunks)[first].y;
  const bool fresh = slot < 0 || p.m.positions[t_first] == 0;
  float S[16][4];
#pragma unroll
  for (int n = 0; n < 16; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = n * 8 + t4 * 2 + (e & 1), v = c0 + g + (e >> 1) * 8;
      S[n][e] = (!fresh && k < K && v < V) ? st[static_cast<long long>(k) * V + v] : 0.f;
    }
  const uint32_t w_base = smem_u32(smem), q_base = w_base + un.q(), b_base = w_base + un.b(), k_base = w_base + un.k();
  const int l7 = lane & 7, l8 = (lane >> 3) & 1, l16 = lane >> 4;
  for (int ci = 0; ci < n_chunks; ++ci) {
    const int4 ch = reinterpret_cast<const int4*>(p.chunks)[first + ci];
    uint32_t uh[4][4], ul[4][4];
    wait(0, ci);
    {                                    // u = U − W S
      float u[8][4];
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float2 x = active ? *reinterpret_cast<const float2*>(sU + (warp * 16 + g + e * 8) * kUPitch + (n * 8 + t4 * 2) * 4) : make_float2(0.f, 0.f);
          u[n][e * 2] = x.x;
          u[n][e * 2 + 1] = x.y;
        }
#pragma unroll
      for (int ks = 0; ks < 8; ++ks) {
        if (ks >= kdk) break;
        uint32_t sh[4], sl[4];
        operand(S[2 * ks], S[2 * ks + 1], sh, sl);
        const int row = ks * 16 + l7 + l8 * 8;
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          uint32_t bh[4], bl[4];
          const uint32_t at = w_base + row * 128 + (((np * 2 + l16) ^ (row & 7)) << 4);
          ldsm4t(at, bh);
          ldsm4t(at + half, bl);
          mma(u[2 * np], sh, bh[0], bh[1]);
          mma(u[2 * np + 1], sh, bh[2], bh[3]);
          mma(u[2 * np], sh, bl[0], bl[1]);
          mma(u[2 * np + 1], sh, bl[2], bl[3]);
          mma(u[2 * np], sl, bh[0], bh[1]);
          mma(u[2 * np + 1], sl, bh[2], bh[3]);
        }
      }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) operand(u[2 * ks], u[2 * ks + 1], uh[ks], ul[ks]);
    }
    __syncthreads();
    if (tid == 0 && ci + 1 < n_chunks && !*abort_flag) load_w(ci + 1);
    wait(1, ci);
    {                                    // outputs
      float o[8][4];
#pragma unroll
      for (int n = 0; n < 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < 8; ++ks) {
        if (ks >= kdk) break;
        uint32_t sh[4], sl[4];
        operand(S[2 * ks], S[2 * ks + 1], sh, sl);
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          uint32_t bh[4], bl[4];
          const int row = np * 16 + l7 + l16 * 8;
          const uint32_t at = q_base + row * KR * 2 + (((ks * 2 + l8) ^ (row & 7)) << 4);
          ldsm4(at, bh);
          ldsm4(at + half, bl);
          mma(o[2 * np], sh, bh[0], bh[1]);
          mma(o[2 * np + 1], sh, bh[2], bh[3]);
          mma(o[2 * np], sh, bl[0], bl[1]);
          mma(o[2 * np + 1], sh, bl[2], bl[3]);
          mma(o[2 * np], sl, bh[0], bh[1]);
          mma(o[2 * np + 1], sl, bh[2], bh[3]);
        }
      }
#pragma unroll
      for (int np = 0; np < 4; ++np)
#pragma unroll
        for (int ks = 0; ks <= np; ++ks) {
          uint32_t bh[4], bl[4];
          const int row = np * 16 + l7 + l16 * 8;
          const uint32_t at = b_base + row * 128 + (((ks * 2 + l8) ^ (row & 7)) << 4);
          ldsm4(at, bh);
          ldsm4(at + 8192, bl);
          mma(o[2 * np], uh[ks], bh[0], bh[1]);
          mma(o[2 * np + 1], uh[ks], bh[2], bh[3]);
          mma(o[2 * np], uh[ks], bl[0], bl[1]);
          mma(o[2 * np + 1], uh[ks], bl[2], bl[3]);
          mma(o[2 * np], ul[ks], bh[0], bh[1]);
          mma(o[2 * np + 1], ul[ks], bh[2], bh[3]);
        }
      // rows of 16 columns per token in the warp's own corner of shared memory, then 16-byte stores
      uint8_t* mine = stage + warp * 2048;
#pragma unroll
      for (int np = 0; np < 4; ++np)
        stsm4t(smem_u32(mine + ((np * 2 + l16) * 8 + l7) * 32 + l8 * 16), pack2(o[2 * np][0], o[2 * np][1]), pack2(o[2 * np][2], o[2 * np][3]),
               pack2(o[2 * np + 1][0], o[2 * np + 1][1]), pack2(o[2 * np + 1][2], o[2 * np + 1][3]));
      __syncwarp();
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = (i * 32 + lane) >> 1, c = c0 + (lane & 1) * 8;
        if (active && ch.y + r < ch.z && c < V)
          *reinterpret_cast<uint4*>(p.out + static_cast<long long>(ch.y + r) * H * V + h * V + c) = *reinterpret_cast<const uint4*>(mine + r * 32 + (lane & 1) * 16);
      }
    }
    __syncthreads();
    if (tid == 0 && ci + 1 < n_chunks && !*abort_flag) load_q(ci + 1);
    wait(2, ci);
    {                                    // S ← decay · S + Σ k uᵀ
      const float* dec = reinterpret_cast<const float*>(smem + un.decay());
#pragma unroll
      for (int n = 0; n < 16; ++n) {
        if (n >= 2 * kdk) break;
        const float2 d = *reinterpret_cast<const float2*>(dec + n * 8 + t4 * 2);
        S[n][0] *= d.x; S[n][1] *= d.y; S[n][2] *= d.x; S[n][3] *= d.y;
      }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        const int row = ks * 16 + l7 + l8 * 8;
#pragma unroll
        for (int np = 0; np < 8; ++np) {
          if (np >= kdk) break;
          uint32_t bh[4], bl[4];
          const uint32_t at = k_base + row * KR * 2 + (((np * 2 + l16) ^ (row & 7)) << 4);
          ldsm4t(at, bh);
          ldsm4t(at + half, bl);
          mma(S[2 * np], uh[ks], bh[0], bh[1]);
          mma(S[2 * np + 1], uh[ks], bh[2], bh[3]);
          mma(S[2 * np], uh[ks], bl[0], bl[1]);
          mma(S[2 * np + 1], uh[ks], bl[2], bl[3]);
          mma(S[2 * np], ul[ks], bh[0], bh[1]);
          mma(S[2 * np + 1], ul[ks], bh[2], bh[3]);
        }
      }
    }
    __syncthreads();
    if (tid == 0 && ci + 1 < n_chunks && !*abort_flag) load_k(ci + 1);
  }
  if (slot < 0 || *abort_flag) return;
#pragma unroll
  for (int n = 0; n < 16; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = n * 8 + t4 * 2 + (e & 1), v = c0 + g + (e >> 1) * 8;
      if (k < K && v < V) st[static_cast<long long>(k) * V + v] = S[n][e];
    }
}

template <int NW>
static cudaError_t scan(const Args& a, int n_parts, cudaStream_t s) {
  static bool once = false;
  if (!once) {
    const cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(scan_bytes(Unit{128, 128}, NW)));
    if (e != cudaSuccess) return e;
    once = true;
  }
  return launch_pdl(delta_scan_kernel<NW>, dim3((a.unit.VP / 16 + NW - 1) / NW, a.m.H, n_parts), dim3(32 * NW), scan_bytes(a.unit, NW), s, a);
}

static Unit unit_of(int K, int V) { return Unit{(K + 63) / 64 * 64, (V + 15) / 16 * 16}; }

}  // namespace dc
}  // namespace mb

using namespace mb;
using namespace mb::dc;

extern "C" long long mb_delta_chunk_bytes(int K, int V) { return unit_of(K, V).bytes(); }

extern "C" int mb_delta_chunk(const void* proj, long long ld, const void* act, MbDelta m, const int* chunks, const int* parts, void* scratch, void* out,
                              int n_chunks, int n_parts, int warps, int* error_flag, cudaStream_t s) {
  if (n_chunks <= 0 || n_parts <= 0) return 0;
  if (m.K % 8 || m.V % 8 || m.K > 128 || m.V > 128 || m.K <= 0 || m.V <= 0 || m.G <= 0 || m.H % m.G || m.raw_ld % 8 || n_chunks > 65535 || n_parts > 65535 ||
      m.H > 65535 || (reinterpret_cast<uintptr_t>(m.raw) | reinterpret_cast<uintptr_t>(m.dt_bias) | reinterpret_cast<uintptr_t>(act)) % 16)
    return -3;
  static bool once = false;
  if (!once) {
    const cudaError_t e = cudaFuncSetAttribute(delta_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(sizeof(Shared)));
    if (e != cudaSuccess) return static_cast<int>(e);
    once = true;
  }
  Args a{reinterpret_cast<const bf16*>(proj), ld, reinterpret_cast<const bf16*>(act), m, chunks, parts, reinterpret_cast<uint8_t*>(scratch), unit_of(m.K, m.V),
         reinterpret_cast<bf16*>(out), error_flag};
  cudaError_t e = launch_pdl(delta_prepare_kernel, dim3(m.H, n_chunks), dim3(kThreads), sizeof(Shared), s, a);
  if (e == cudaSuccess) e = warps >= 8 ? scan<8>(a, n_parts, s) : warps >= 4 ? scan<4>(a, n_parts, s) : scan<2>(a, n_parts, s);
  return static_cast<int>(e);
}
