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

int make_tmap_bf16_2d(CUtensorMap* out, const void* base, long long rows, long long cols, long long ld, int box_rows, int box_cols);

namespace dc {

using mx::bf16;
static constexpr int C = 64, kThreads = 512;
static constexpr int P = 136, LP = 132, AP = 72, DP = 20;      // shared rows: bf16 tiles (≤ 128 wide), floats per channel, bf16 per token, floats of a diagonal block
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
  bf16 a_hi[C * AP], a_lo[C * AP];         // A below its diagonal blocks, their inverses T in these
  float diagonal[4][16 * DP];              // A inside them
  float D[4][128], before[4][128], after[4][128], between[7][128];
  float fq[C], fk[C], beta[C], beta_k[C];
  int direct[4];
  uint64_t full;             // the inputs of a unit have come
};

// Pairs of blocks i: the diagonal ones, those with blocks between them, neighbours.  The first seven have a factor on the columns, between[i].
__device__ __forceinline__ void pair_of(int i, int& a, int& b) {
  a = i < 4 ? i : i < 7 ? (i == 4 ? 2 : 3) : i - 6;
  b = i < 4 ? i : i < 7 ? (i == 6 ? 1 : 0) : i - 7;
}

__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
// 1 / √x: the approximation and one Newton step, good to the last bits
__device__ __forceinline__ float inv_sqrt(float x) {
  const float y = rsqrtf(x);
  return y * fmaf(-0.5f * x, y * y, 1.5f);
}

// A CTA per SM takes every gridDim.x-th (chunk, head).  The inputs of the next one come by TMA while the products of the last phase run, into
// tiles that are free by then: boxes of 64 tokens × 64 columns (128-byte swizzle), q and v over q_hi and q_lo, k and what decays come from
// over c_hi and c_lo.  Rows behind the chunk and columns behind the head are whatever lies there: they count as zeros.
__global__ void __launch_bounds__(kThreads, 1) delta_prepare_kernel(const __grid_constant__ CUtensorMap tm_act, const __grid_constant__ CUtensorMap tm_raw,
                                                                    Args p, int n_units) {
  extern __shared__ __align__(1024) uint8_t smem[];
  Shared& s = *reinterpret_cast<Shared*>(smem);
  if (smem_u32(smem) & 1023u) {
    if (threadIdx.x == 0) atomicExch(p.error_flag, 93);
    return;
  }
  const int H = p.m.H, K = p.m.K, V = p.m.V, per = H / p.m.G, CH = 2 * p.m.G * K + H * V;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int kdk = (K + 15) / 16, kdv = (V + 15) / 16;
  const int KR = p.unit.KR, half = p.unit.half();
  const float q_scale = __fdiv_rn(1.f, __fsqrt_rn(static_cast<float>(K)));
  const int my_row = tid >> 4, my_c = (tid & 15) * 8;      // 8 channels of rows my_row and my_row + 32
  if (tid == 0) {
    mbar_init(&s.full, 1);
    mbar_fence_init();
  }
  pdl_trigger();
  pdl_wait();
  __syncthreads();
  // what a thread keeps of the next unit: its chunk, its channels' bias, its row's β, the head's rate
  int4 ch = reinterpret_cast<const int4*>(p.chunks)[blockIdx.x / H];
  uint4 bias_raw = make_uint4(0, 0, 0, 0);
  bf16 beta_raw = __float2bfloat16(0.f), a_raw = __float2bfloat16(0.f);
  uint8_t* in_q = reinterpret_cast<uint8_t*>(s.q_hi);      // [q | v], then [k | raw]: two boxes each
  uint8_t* in_k = reinterpret_cast<uint8_t*>(s.c_hi);
  auto fetch = [&](int idx) {
    const int h = idx % H, gq = h / per;
    if (tid == 0) {
      const int na = (K + 63) / 64, nv = (V + 63) / 64;
      mbar_expect_tx(&s.full, (3 * na + nv) * 8192);
      for (int i = 0; i < na; ++i) {
        tma_load_2d(in_q + i * 8192, &tm_act, &s.full, gq * K + i * 64, ch.y);
        tma_load_2d(in_k + i * 8192, &tm_act, &s.full, (p.m.G + gq) * K + i * 64, ch.y);
        tma_load_2d(in_k + 16384 + i * 8192, &tm_raw, &s.full, h * K + i * 64, ch.y);
      }
      for (int i = 0; i < nv; ++i) tma_load_2d(in_q + 16384 + i * 8192, &tm_act, &s.full, 2 * p.m.G * K + h * V + i * 64, ch.y);
    }
    if (my_c < K) bias_raw = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(p.m.dt_bias) + h * K + my_c);
    a_raw = reinterpret_cast<const bf16*>(p.m.A_log)[h];
    if (tid < ch.z - ch.y) beta_raw = p.proj[(ch.y + tid) * p.ld + p.m.beta_at + h];      // (at most 64 tokens)
  };
  fetch(blockIdx.x);
  uint32_t phase = 0;
  for (int idx = blockIdx.x; idx < n_units; idx += gridDim.x) {
    const int h = idx % H, gq = h / per, t0_now = ch.y, n_now = ch.z - ch.y, after_idx = idx + gridDim.x;
    if (after_idx < n_units) ch = reinterpret_cast<const int4*>(p.chunks)[after_idx / H];
    uint8_t* unit = p.scratch + static_cast<long long>(idx) * p.unit.bytes();
    if (!mbar_wait(&s.full, phase)) {
      atomicExch(p.error_flag, 92);
      return;
    }
    phase ^= 1;
    __syncthreads();
    // ---- q and k with the factors that make unit vectors of them, v into its place, log decays, β
    uint4 q_in[2], k_in[2];
    const float rate = __expf(__bfloat162float(a_raw));
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = my_row + i * 32, at = r * P + my_c;
      const int from = (my_c >> 6) * 8192 + r * 128 + ((((my_c >> 3) & 7) ^ (r & 7)) << 4);
      const bool ok = r < n_now && my_c < K;
      uint4 v = make_uint4(0, 0, 0, 0), x = make_uint4(0, 0, 0, 0);
      q_in[i] = k_in[i] = v;
      if (ok) {
        q_in[i] = *reinterpret_cast<const uint4*>(in_q + from);
        k_in[i] = *reinterpret_cast<const uint4*>(in_k + from);
        x = *reinterpret_cast<const uint4*>(in_k + 16384 + from);
      }
      if (r < n_now && my_c < V) v = *reinterpret_cast<const uint4*>(in_q + 16384 + from);
      *reinterpret_cast<uint4*>(s.v + at) = v;
      const uint32_t qw[4] = {q_in[i].x, q_in[i].y, q_in[i].z, q_in[i].w}, kw[4] = {k_in[i].x, k_in[i].y, k_in[i].z, k_in[i].w};
      float sq = 0.f, sk = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        sq += lo16(qw[j]) * lo16(qw[j]) + hi16(qw[j]) * hi16(qw[j]);
        sk += lo16(kw[j]) * lo16(kw[j]) + hi16(kw[j]) * hi16(kw[j]);
      }
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) {    // a row's 16 threads are half a warp
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
      }
      if (my_c == 0) {
        s.fq[r] = inv_sqrt(sq + 1e-6f) * q_scale;
        s.fk[r] = inv_sqrt(sk + 1e-6f);
      }
      const uint32_t xw[4] = {x.x, x.y, x.z, x.w}, bw[4] = {bias_raw.x, bias_raw.y, bias_raw.z, bias_raw.w};
      float l[8];
#pragma unroll
      for (int j = 0; j < 8; ++j)
        l[j] = ok ? -rate * softplus2((j & 1) ? hi16(xw[j / 2]) + hi16(bw[j / 2]) : lo16(xw[j / 2]) + lo16(bw[j / 2])) : 0.f;
      mx::store_n<8>(s.L + r * LP + my_c, l);
    }
    if (tid < C) s.beta[tid] = tid < n_now ? mx::sigmoid_t<bf16>(__bfloat162float(beta_raw)) : 0.f;
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
      s.between[0][tid] = e2(fminf(-d0, -kFar));           // blocks beyond are summed directly
      s.between[1][tid] = e2(fminf(-d1, -kFar));
      s.between[2][tid] = e2(fminf(-d2, -kFar));
      s.between[3][tid] = e2(fminf(-d3, -kFar));
      s.between[4][tid] = e2(d1);
      s.between[5][tid] = e2(d1 + d2);
      s.between[6][tid] = e2(d2);
      reinterpret_cast<float*>(unit + p.unit.decay())[tid] = e2(d0 + d1 + d2 + d3);
    } else if (tid < 128 + C) {
      s.beta_k[tid - 128] = s.beta[tid - 128] * s.fk[tid - 128];
    }
    __syncthreads();
    // ---- q and k decayed from the start of their block, k to its end; queries decayed from the chunk's start, keys to its end
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = my_row + i * 32, c = my_c, at = r * P + c;
      float q[8], k[8], l[8], d[8], x[8];
      uint4 hi, lo;
      const uint32_t qw[4] = {q_in[i].x, q_in[i].y, q_in[i].z, q_in[i].w}, kw[4] = {k_in[i].x, k_in[i].y, k_in[i].z, k_in[i].w};
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        q[j] = (j & 1) ? hi16(qw[j / 2]) : lo16(qw[j / 2]);
        k[j] = (j & 1) ? hi16(kw[j / 2]) : lo16(kw[j / 2]);
      }
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
      if (c < kdk * 16) {
        float f[8];
        mx::load_n<8>(s.before[r >> 4] + c, f);
        const float scale = s.fq[r];
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] *= f[j] * scale;
        split8(x, hi, lo);
        uint8_t* to = unit + p.unit.q() + r * KR * 2 + (((c >> 3) ^ (r & 7)) << 4);
        *reinterpret_cast<uint4*>(to) = hi;
        *reinterpret_cast<uint4*>(to + half) = lo;
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] = k[j] * l[j];
      split8(x, hi, lo);
      *reinterpret_cast<uint4*>(s.k_hi + at) = hi;
      *reinterpret_cast<uint4*>(s.k_lo + at) = lo;
      split8(d, hi, lo);
      *reinterpret_cast<uint4*>(s.c_hi + at) = hi;
      *reinterpret_cast<uint4*>(s.c_lo + at) = lo;
      if (c < kdk * 16) {
        float f[8];
        mx::load_n<8>(s.after[r >> 4] + c, f);
        const float scale = s.fk[r];
#pragma unroll
        for (int j = 0; j < 8; ++j) d[j] *= f[j] * scale;
        split8(d, hi, lo);
        uint8_t* to = unit + p.unit.k() + r * KR * 2 + (((c >> 3) ^ (r & 7)) << 4);
        *reinterpret_cast<uint4*>(to) = hi;
        *reinterpret_cast<uint4*>(to + half) = lo;
      }
    }
    __syncthreads();
    // ---- A and B, a warp per pair of blocks; the diagonal blocks of I + A are inverted by the warps that made them
    if (warp < 10) {
      int a, b;
      pair_of(warp, a, b);
      float kk[2][4] = {}, qk[2][4] = {}, kk1[2][4] = {}, qk1[2][4] = {};      // (the products with low parts have sums of their own)
      if (a == b && s.direct[a]) {
#pragma unroll 1
        for (int x = 0; x < 8; ++x) {
          const int i = a * 16 + g + (x & 2) * 4, j = a * 16 + (x >> 2) * 8 + t4 * 2 + (x & 1);
          float sk = 0.f, sq = 0.f;
          if (j <= i && i < n_now) {
            const bf16* qi = p.act + static_cast<long long>(t0_now + i) * CH + gq * K;
            const bf16* ki = qi + p.m.G * K;
            const bf16* kj = p.act + static_cast<long long>(t0_now + j) * CH + p.m.G * K + gq * K;
            for (int c = 0; c < K; ++c) {
              const float w = __bfloat162float(kj[c]) * e2(s.L[i * LP + c] - s.L[j * LP + c]);
              sk = fmaf(__bfloat162float(ki[c]), w, sk);
              sq = fmaf(__bfloat162float(qi[c]), w, sq);
            }
          }
#pragma unroll
          for (int y = 0; y < 8; ++y)
            if (y == x) { kk[y >> 2][y & 3] = sk; qk[y >> 2][y & 3] = sq; }
        }
        __syncwarp();
      } else {
        const int row_a = (a * 16 + (lane & 15)) * P + (lane >> 4) * 8;
        const int row_b = (b * 16 + (lane & 7) + ((lane >> 4) << 3)) * P + ((lane >> 3) & 1) * 8;
        const float* fac = s.between[min(warp, 6)];
#pragma unroll 2
        for (int ks = 0; ks < kdk; ++ks) {
          uint32_t qh[4], ql[4], kh[4], kl[4], ch[4], cl[4];
          ldsm4(smem_u32(s.c_hi + row_b + ks * 16), ch);
          ldsm4(smem_u32(s.c_lo + row_b + ks * 16), cl);
          ldsm4(smem_u32(s.k_hi + row_a + ks * 16), kh);
          ldsm4(smem_u32(s.q_hi + row_a + ks * 16), qh);
          ldsm4(smem_u32(s.k_lo + row_a + ks * 16), kl);
          ldsm4(smem_u32(s.q_lo + row_a + ks * 16), ql);
          if (warp < 7) {
#pragma unroll
            for (int i = 0; i < 2; ++i) {
              const float2 f = *reinterpret_cast<const float2*>(fac + ks * 16 + i * 8 + t4 * 2);
#pragma unroll
              for (int n = 0; n < 4; n += 2) split2((lo16(ch[n + i]) + lo16(cl[n + i])) * f.x, (hi16(ch[n + i]) + hi16(cl[n + i])) * f.y, ch[n + i], cl[n + i]);
            }
          }
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            mma(kk[n], kh, ch[2 * n], ch[2 * n + 1]);
            mma(qk[n], qh, ch[2 * n], ch[2 * n + 1]);
          }
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            mma(kk1[n], kh, cl[2 * n], cl[2 * n + 1]);
            mma(qk1[n], qh, cl[2 * n], cl[2 * n + 1]);
          }
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            mma(kk1[n], kl, ch[2 * n], ch[2 * n + 1]);
            mma(qk1[n], ql, ch[2 * n], ch[2 * n + 1]);
          }
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int i = a * 16 + g + e * 4, j = b * 16 + n * 8 + t4 * 2;
          const float k0 = kk[n][e] + kk1[n][e], k1 = kk[n][e + 1] + kk1[n][e + 1], q0 = qk[n][e] + qk1[n][e], q1 = qk[n][e + 1] + qk1[n][e + 1];
          const float f0 = s.fk[j], f1 = s.fk[j + 1], fi = s.beta_k[i], fo = s.fq[i];
          uint32_t hi, lo;
          if (a == b) {
            *reinterpret_cast<float2*>(s.diagonal[a] + (i & 15) * DP + (j & 15)) = make_float2(k0 * fi * f0, k1 * fi * f1);      // (read below its diagonal)
          } else {
            split2(k0 * fi * f0, k1 * fi * f1, hi, lo);
            *reinterpret_cast<uint32_t*>(s.a_hi + i * AP + j) = hi;
            *reinterpret_cast<uint32_t*>(s.a_lo + i * AP + j) = lo;
          }
          split2(j <= i ? q0 * fo * f0 : 0.f, j + 1 <= i ? q1 * fo * f1 : 0.f, hi, lo);
          uint8_t* at = unit + p.unit.b() + i * 128 + (((j >> 3) ^ (i & 7)) << 4) + (j & 7) * 2;
          *reinterpret_cast<uint32_t*>(at) = hi;
          *reinterpret_cast<uint32_t*>(at + 8192) = lo;
        }
    }
    if (warp < 4) {                        // a lane per column of the inverse
      __syncwarp();
      const int c = lane & 15;
      const float* blk = s.diagonal[warp];
      float x[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float r[4] = {i == c ? 1.f : 0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int j = 0; j < i; j += 4) {
          const float4 a = *reinterpret_cast<const float4*>(blk + i * DP + j);
          r[0] = fmaf(-a.x, x[j], r[0]);
          if (j + 1 < i) r[1] = fmaf(-a.y, x[j + 1], r[1]);
          if (j + 2 < i) r[2] = fmaf(-a.z, x[j + 2], r[2]);
          if (j + 3 < i) r[3] = fmaf(-a.w, x[j + 3], r[3]);
        }
        x[i] = (r[0] + r[1]) + (r[2] + r[3]);
      }
      if (lane < 16) {
        const int at = warp * 16 * AP + warp * 16 + c;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const bf16 hi = __float2bfloat16(x[i]);
          s.a_hi[at + i * AP] = hi;
          s.a_lo[at + i * AP] = __float2bfloat16(x[i] - __bfloat162float(hi));
        }
      }
    }
    fence_proxy_async();                   // what was written to the tiles comes before the copies into them
    __syncthreads();
    if (after_idx < n_units) fetch(after_idx);
    // ---- X = T·[β v | β k e^G] by blocks of tokens, transposed: a warp's 16 columns are the rows of its products
    const int a_row = (lane & 7) + ((lane >> 4) << 3), a_col = ((lane >> 3) & 1) * 8;
    const int r_row = (lane & 7) + ((lane >> 4) << 3), r_col = ((lane >> 3) & 1) * 8;
    for (int mt = warp; mt < kdv + kdk; mt += kThreads / 32) {
      const bool is_u = mt < kdv;
      const int c0 = (is_u ? mt : mt - kdv) * 16;
      uint8_t* w_rows = reinterpret_cast<uint8_t*>(s.L) + (mt - kdv) % 8 * 4096;      // 16 rows of W, hi and lo, on their way out (the decays are not needed any more)
      uint32_t xh[4][4], xl[4][4];
#pragma unroll
      for (int a = 0; a < 4; ++a) {
        float acc[2][4], acc1[2][4];
        // rows of A (or T) are the columns of the second factor; the products with low parts have sums of their own
        auto times = [&](const uint32_t (&yh)[4], const uint32_t (&yl)[4], int b) {
          uint32_t bh[4], bl[4];
          const int at = (a * 16 + a_row) * AP + b * 16 + a_col;
          ldsm4(smem_u32(s.a_hi + at), bh);
          ldsm4(smem_u32(s.a_lo + at), bl);
          mma(acc[0], yh, bh[0], bh[1]);
          mma(acc[1], yh, bh[2], bh[3]);
          mma(acc1[0], yh, bl[0], bl[1]);
          mma(acc1[1], yh, bl[2], bl[3]);
          mma(acc1[0], yl, bh[0], bh[1]);
          mma(acc1[1], yl, bh[2], bh[3]);
        };
        auto clear = [&]() {
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[n][e] = acc1[n][e] = 0.f;
        };
        auto sum = [&]() {
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[n][e] += acc1[n][e];
        };
        clear();
#pragma unroll
        for (int b = 0; b < a; ++b) times(xh[b], xl[b], b);
        sum();
        // the block's right-hand side, transposed on its way from shared memory: register 2n + e holds tokens 8n + 2·t4 and the next of column g + 8e
        const int at = (a * 16 + r_row) * P + c0 + r_col;
        if (is_u) {
          uint32_t v[4];
          ldsm4t(smem_u32(s.v + at), v);
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const float2 f = *reinterpret_cast<const float2*>(s.beta + a * 16 + n * 8 + t4 * 2);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              acc[n][e * 2] = fmaf(lo16(v[n * 2 + e]), f.x, -acc[n][e * 2]);
              acc[n][e * 2 + 1] = fmaf(hi16(v[n * 2 + e]), f.y, -acc[n][e * 2 + 1]);
            }
          }
        } else {
          uint32_t v[4], w[4];
          ldsm4t(smem_u32(s.k_hi + at), v);
          ldsm4t(smem_u32(s.k_lo + at), w);
          const float from[2] = {s.before[a][c0 + g], s.before[a][c0 + g + 8]};
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const float2 f = *reinterpret_cast<const float2*>(s.beta_k + a * 16 + n * 8 + t4 * 2);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              acc[n][e * 2] = fmaf(lo16(v[n * 2 + e]) + lo16(w[n * 2 + e]), f.x * from[e], -acc[n][e * 2]);
              acc[n][e * 2 + 1] = fmaf(hi16(v[n * 2 + e]) + hi16(w[n * 2 + e]), f.y * from[e], -acc[n][e * 2 + 1]);
            }
          }
        }
        uint32_t yh[4], yl[4];
        operand(acc[0], acc[1], yh, yl);
        clear();
        times(yh, yl, a);
        sum();
        operand(acc[0], acc[1], xh[a], xl[a]);
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int c = c0 + g + e * 8, t = a * 16 + n * 8 + t4 * 2;
            if (is_u) {
              *reinterpret_cast<float2*>(unit + p.unit.u() + c * kUPitch + t * 4) = make_float2(acc[n][e * 2], acc[n][e * 2 + 1]);
            } else {                       // −W: the second kernel adds
              uint8_t* to = w_rows + (g + e * 8) * 128 + (((t >> 3) ^ (c & 7)) << 4) + (t & 7) * 2;
              *reinterpret_cast<uint32_t*>(to) = xh[a][n * 2 + e] ^ 0x80008000u;
              *reinterpret_cast<uint32_t*>(to + 2048) = xl[a][n * 2 + e] ^ 0x80008000u;
            }
          }
      }
      if (!is_u) {
        __syncwarp();
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int at = (i * 32 + lane) * 16;
          *reinterpret_cast<uint4*>(unit + c0 * 128 + at) = *reinterpret_cast<const uint4*>(w_rows + at);
          *reinterpret_cast<uint4*>(unit + half + c0 * 128 + at) = *reinterpret_cast<const uint4*>(w_rows + 2048 + at);
        }
        __syncwarp();
      }
    }
  }
}

// the warps' corners: outputs on their way out, and with two warps per 16 columns the parts they exchange
__host__ __device__ constexpr int corner_bytes(int ks) { return ks == 2 ? 4096 + 128 : 2048; }
static size_t scan_bytes(const Unit& u, int nw, int ks) { return static_cast<size_t>(u.u()) + nw * 16 * kUPitch + nw * ks * corner_bytes(ks) + 64; }

// c[2·np], c[2·np + 1] += (ah + al)·(hi + lo) without the product of the low parts; b[np] = the operands of two neighbouring accumulators.  One
// accumulator comes up again only after all others.
template <int N>
__device__ __forceinline__ void products(float (*c)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[N][4], const uint32_t (&bl)[N][4]) {
#pragma unroll
  for (int n = 0; n < N; ++n) {
    mma(c[2 * n], ah, bh[n][0], bh[n][1]);
    mma(c[2 * n + 1], ah, bh[n][2], bh[n][3]);
  }
#pragma unroll
  for (int n = 0; n < N; ++n) {
    mma(c[2 * n], ah, bl[n][0], bl[n][1]);
    mma(c[2 * n + 1], ah, bl[n][2], bl[n][3]);
  }
#pragma unroll
  for (int n = 0; n < N; ++n) {
    mma(c[2 * n], al, bh[n][0], bh[n][1]);
    mma(c[2 * n + 1], al, bh[n][2], bh[n][3]);
  }
}

// grid (slices of 16·NW value columns, heads, parts of sequences), 32·NW·KS threads.  KS = 2: two warps share 16 value columns, each with half
// of the channels; they exchange their parts of u and of the outputs.
template <int NW, int KS>
__global__ void __launch_bounds__(32 * NW * KS, 1) delta_scan_kernel(Args p) {
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int NT = 16 / KS, KT = 8 / KS;               // accumulators (8 channels) and k steps (16 channels) of a warp
  const Unit un = p.unit;
  const int KR = un.KR, half = un.half();
  uint8_t* sU = smem + un.u();
  uint8_t* corners = sU + NW * 16 * kUPitch;
  uint64_t* bars = reinterpret_cast<uint64_t*>(corners + NW * KS * corner_bytes(KS));        // W, q and U | B, k and decay
  volatile int* abort_flag = reinterpret_cast<volatile int*>(bars + 2);
  const int h = blockIdx.y, H = p.m.H, K = p.m.K, V = p.m.V, kdk = (K + 15) / 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int cg = warp % NW, kh = warp / NW, ks0 = kh * KT;
  if (tid == 0) {
    for (int i = 0; i < 2; ++i) mbar_init(&bars[i], 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  pdl_trigger();
  pdl_wait();
  const int4 part = reinterpret_cast<const int4*>(p.parts)[blockIdx.z];
  const int first = part.x, n_chunks = part.y, slot = p.m.slots[part.z];
  const int c_cta = blockIdx.x * NW * 16, c0 = c_cta + cg * 16;
  const int u_rows = min(NW * 16, un.VP - c_cta);
  const bool active = c0 < un.VP;        // (the last slice may be narrower)
  __syncthreads();
  auto unit_of = [&](int i) { return p.scratch + (static_cast<long long>(first + i) * H + h) * un.bytes(); };
  auto load_first = [&](int i) {
    const uint8_t* src = unit_of(i);
    mbar_expect_tx(&bars[0], 4 * half + u_rows * kUPitch);
    bulk_load(smem, src, 4 * half, &bars[0]);
    bulk_load(sU, src + un.u() + c_cta * kUPitch, u_rows * kUPitch, &bars[0]);
  };
  auto load_second = [&](int i) {
    const uint32_t bytes = un.u() - un.b();
    mbar_expect_tx(&bars[1], bytes);
    bulk_load(smem + un.b(), unit_of(i) + un.b(), bytes, &bars[1]);
  };
  if (tid == 0) {
    load_first(0);
    load_second(0);
  }
  auto wait = [&](int which, int i) {
    if (*abort_flag) return;
    if (!mbar_wait(&bars[which], i & 1)) {
      *abort_flag = 1;
      atomicExch(p.error_flag, 91);
    }
  };
  // Sᵀ: rows are the warp's value columns g and g + 8, accumulator n holds channels 16·ks0 + 8n + 2·t4 and the next
  float* st = p.m.state + (static_cast<long long>(max(slot, 0)) * H + h) * K * V;
  const int t_first = reinterpret_cast<const int4*>(p.chunks)[first].y;
  const bool fresh = slot < 0 || p.m.positions[t_first] == 0;
  float S[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = ks0 * 16 + n * 8 + t4 * 2 + (e & 1), v = c0 + g + (e >> 1) * 8;
      S[n][e] = (!fresh && k < K && v < V) ? st[static_cast<long long>(k) * V + v] : 0.f;
    }
  const uint32_t w_base = smem_u32(smem), q_base = w_base + un.q(), b_base = w_base + un.b(), k_base = w_base + un.k();
  const int l7 = lane & 7, l8 = (lane >> 3) & 1, l16 = lane >> 4;
  uint8_t* mine = corners + warp * corner_bytes(KS);
  uint8_t* other = corners + (warp < NW ? warp + NW : warp - NW) * corner_bytes(KS);
  auto pair_sync = [&]() { asm volatile("bar.sync %0, 64;" ::"r"(cg + 1) : "memory"); };
  // accumulators [n0, n0 + N) of a warp in its corner and back: a lane's float4s, 32 lanes side by side
  auto put = [&](const float (*x)[4], int n0, int N) {
#pragma unroll
    for (int n = 0; n < 8; ++n)
      if (n < N) *reinterpret_cast<float4*>(mine + (n * 32 + lane) * 16) = make_float4(x[n0 + n][0], x[n0 + n][1], x[n0 + n][2], x[n0 + n][3]);
  };
  auto take = [&](float (*x)[4], int n0, int N) {
#pragma unroll
    for (int n = 0; n < 8; ++n)
      if (n < N) {
        const float4 v = *reinterpret_cast<const float4*>(other + (n * 32 + lane) * 16);
        x[n0 + n][0] += v.x; x[n0 + n][1] += v.y; x[n0 + n][2] += v.z; x[n0 + n][3] += v.w;
      }
  };
  for (int ci = 0; ci < n_chunks; ++ci) {
    const int4 ch = reinterpret_cast<const int4*>(p.chunks)[first + ci];
    uint32_t uh[4][4], ul[4][4];
    float o[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    wait(0, ci);
    {                                    // u = U − W S, o = q S
      float u[8][4];
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float2 x = make_float2(0.f, 0.f);
          if (active && kh == 0) x = *reinterpret_cast<const float2*>(sU + (cg * 16 + g + e * 8) * kUPitch + (n * 8 + t4 * 2) * 4);
          u[n][e * 2] = x.x;
          u[n][e * 2 + 1] = x.y;
        }
#pragma unroll
      for (int i = 0; i < KT; ++i) {
        if (ks0 + i >= kdk) break;
        uint32_t sh[4], sl[4], bh[4][4], bl[4][4];
        operand(S[2 * i], S[2 * i + 1], sh, sl);
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          const int row = (ks0 + i) * 16 + l7 + l8 * 8;
          const uint32_t at = w_base + row * 128 + (((np * 2 + l16) ^ (row & 7)) << 4);
          ldsm4t(at, bh[np]);
          ldsm4t(at + half, bl[np]);
        }
        products<4>(u, sh, sl, bh, bl);
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          const int row = np * 16 + l7 + l16 * 8;
          const uint32_t at = q_base + row * KR * 2 + ((((ks0 + i) * 2 + l8) ^ (row & 7)) << 4);
          ldsm4(at, bh[np]);
          ldsm4(at + half, bl[np]);
        }
        products<4>(o, sh, sl, bh, bl);
      }
      if (KS == 2) {
        put(u, 0, 8);
        pair_sync();
        take(u, 0, 8);
      }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) operand(u[2 * ks], u[2 * ks + 1], uh[ks], ul[ks]);
    }
    __syncthreads();
    if (tid == 0 && ci + 1 < n_chunks && !*abort_flag) load_first(ci + 1);
    wait(1, ci);
    // o += B u, by blocks of 16 tokens; of two warps one takes the last row of blocks
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t bh[4][4], bl[4][4];
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        if (np < ks || (KS == 2 && (np == 3) != (kh == 1))) continue;
        const int row = np * 16 + l7 + l16 * 8;
        const uint32_t at = b_base + row * 128 + (((ks * 2 + l8) ^ (row & 7)) << 4);
        ldsm4(at, bh[np]);
        ldsm4(at + 8192, bl[np]);
      }
#pragma unroll
      for (int term = 0; term < 3; ++term)
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          if (np < ks || (KS == 2 && (np == 3) != (kh == 1))) continue;
          mma(o[2 * np], term == 2 ? ul[ks] : uh[ks], term == 1 ? bl[np][0] : bh[np][0], term == 1 ? bl[np][1] : bh[np][1]);
          mma(o[2 * np + 1], term == 2 ? ul[ks] : uh[ks], term == 1 ? bl[np][2] : bh[np][2], term == 1 ? bl[np][3] : bh[np][3]);
        }
    }
    if (KS == 2) {                       // each finishes half of the tokens
      if (kh == 0) put(o, 4, 4);
      else put(o, 0, 4);
    }
    {                                    // S ← decay · S + Σ k uᵀ
      const float* dec = reinterpret_cast<const float*>(smem + un.decay()) + ks0 * 16;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const float2 d = *reinterpret_cast<const float2*>(dec + n * 8 + t4 * 2);
        S[n][0] *= d.x; S[n][1] *= d.y; S[n][2] *= d.x; S[n][3] *= d.y;
      }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        const int row = ks * 16 + l7 + l8 * 8;
#pragma unroll
        for (int n4 = 0; n4 < KT; n4 += 4) {
          if (ks0 + n4 >= kdk) break;
          uint32_t bh[4][4], bl[4][4];
#pragma unroll
          for (int np = 0; np < 4; ++np) {               // (columns behind K: whatever lies there stays in accumulators that nobody reads)
            const int piece = min((ks0 + n4 + np) * 2 + l16, KR / 8 - 1);
            const uint32_t at = k_base + row * KR * 2 + ((piece ^ (row & 7)) << 4);
            ldsm4t(at, bh[np]);
            ldsm4t(at + half, bl[np]);
          }
          products<4>(S + 2 * n4, uh[ks], ul[ks], bh, bl);
        }
      }
    }
    __syncthreads();
    if (tid == 0 && ci + 1 < n_chunks && !*abort_flag) load_second(ci + 1);
    if (KS == 2) {
      if (kh == 0) take(o, 0, 4);
      else take(o, 4, 4);
      pair_sync();
    }
    // rows of 16 columns per token in the warp's own corner of shared memory, then 16-byte stores
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      if (KS == 2 && (np >> 1) != kh) continue;
      stsm4t(smem_u32(mine + ((np * 2 + l16) * 8 + l7) * 32 + l8 * 16), pack2(o[2 * np][0], o[2 * np][1]), pack2(o[2 * np][2], o[2 * np][3]),
             pack2(o[2 * np + 1][0], o[2 * np + 1][1]), pack2(o[2 * np + 1][2], o[2 * np + 1][3]));
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      if (KS == 2 && (i >> 1) != kh) continue;
      const int r = (i * 32 + lane) >> 1, c = c0 + (lane & 1) * 8;
      if (active && ch.y + r < ch.z && c < V)
        *reinterpret_cast<uint4*>(p.out + static_cast<long long>(ch.y + r) * H * V + h * V + c) = *reinterpret_cast<const uint4*>(mine + r * 32 + (lane & 1) * 16);
    }
    __syncwarp();
  }
  if (slot < 0 || *abort_flag) return;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = ks0 * 16 + n * 8 + t4 * 2 + (e & 1), v = c0 + g + (e >> 1) * 8;
      if (k < K && v < V) st[static_cast<long long>(k) * V + v] = S[n][e];
    }
}

template <int NW, int KS>
static cudaError_t scan(const Args& a, int n_parts, cudaStream_t s) {
  static bool once = false;
  if (!once) {
    const cudaError_t e =
        cudaFuncSetAttribute(delta_scan_kernel<NW, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(scan_bytes(Unit{128, 128}, NW, KS)));
    if (e != cudaSuccess) return e;
    once = true;
  }
  return launch_pdl(delta_scan_kernel<NW, KS>, dim3((a.unit.VP / 16 + NW - 1) / NW, a.m.H, n_parts), dim3(32 * NW * KS), scan_bytes(a.unit, NW, KS), s, a);
}

static Unit unit_of(int K, int V) { return Unit{(K + 63) / 64 * 64, (V + 15) / 16 * 16}; }

}  // namespace dc
}  // namespace mb

using namespace mb;
using namespace mb::dc;

extern "C" long long mb_delta_chunk_bytes(int K, int V) { return unit_of(K, V).bytes(); }

extern "C" int mb_delta_chunk(const void* proj, long long ld, const void* act, MbDelta m, const int* chunks, const int* parts, void* scratch, void* out,
                              int T, int n_chunks, int n_parts, int warps, int* error_flag, cudaStream_t s) {
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
  CUtensorMap tm_act, tm_raw;
  const long long CH = 2ll * m.G * m.K + static_cast<long long>(m.H) * m.V;
  int rc = make_tmap_bf16_2d(&tm_act, act, T, CH, CH, C, 64);
  if (rc) return 1000 + rc;
  rc = make_tmap_bf16_2d(&tm_raw, m.raw, T, static_cast<long long>(m.H) * m.K, m.raw_ld, C, 64);
  if (rc) return 2000 + rc;
  const int n_units = n_chunks * m.H;
  cudaError_t e = launch_pdl(delta_prepare_kernel, dim3(n_units < 148 ? n_units : 148), dim3(kThreads), sizeof(Shared), s, tm_act, tm_raw, a, n_units);
  // with few slices per CTA two warps share one, unless the channels of a second one are all padding
  const bool two = m.K > 64;
  if (e == cudaSuccess)
    e = warps >= 8 ? scan<8, 1>(a, n_parts, s) : warps >= 4 ? (two ? scan<4, 2>(a, n_parts, s) : scan<4, 1>(a, n_parts, s))
                                               : (two ? scan<2, 2>(a, n_parts, s) : scan<2, 1>(a, n_parts, s));
  return static_cast<int>(e);
}
