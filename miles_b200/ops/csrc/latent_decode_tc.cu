// Decode attention over cached latents on tcgen05 tensor cores (bf16, pages of a multiple of 64 tokens).
//
// One CTA = (key split, 32 heads, token).  The KEYS are the 128-row side of the score product and the latent columns the 128-row
// side of the other, the heads are the narrow side of both, so 32 heads fill an instruction:
//     Sᵀ [128 keys, 32]     = C · Qᵀ              C: cached rows (K-major), Q: absorbed queries of 32 heads
//     Oᵀ [128 latent, 32] += Cᵀ · P_hi + Cᵀ · P_lo    per 128 latent columns; the same rows in shared memory, read MN-major
// The softmax weights are two bf16 parts (16 bits of mantissa).  Tiles of 64 keys, brought by TMA page by page, alternate between two
// stages: the upper and the lower half of 128-row shared-memory atoms (64 columns each).  A score product covers both halves; the
// rows of the other stage, valid or in flight, are results that nobody reads.  Each stage has its own softmax warpgroup, running
// maximum, sum and Oᵀ, so the loads, products and softmax of neighbouring tiles overlap; the two are added up at the end.  The atom
// pairs of a stage are refilled one by one as their parts of Oᵀ are done.
//   warp 0       TMA        warp 1      MMA issue, TMEM owner
//   warps 2..9   two warpgroups, thread = row of Sᵀ (softmax of its stage's 64 keys) and = latent column (rescaling, result)
// Keys before the window, after the token or outside the sequence get weight 0; a page-table entry outside the pool reads as zeros.
#include "mixers.cuh"
#include "ptx.cuh"

namespace mb {

int make_tmap_bf16_2d(CUtensorMap* out, const void* base, long long rows, long long cols, long long ld, int box_rows, int box_cols);

namespace ldt {

static constexpr int TK = 64, HT = 32;
static constexpr int kAtom = 2 * TK * 128, kQAtom = HT * 128, kPBytes = TK * 128;  // bytes: 64 columns of both stages / of the queries; P of a stage
static constexpr uint32_t kTmemCols = 512;                                         // Sᵀ: 4 × 32 columns per stage; Oᵀ: 4 × 32 per stage
// A product of 32 columns is shorter than its own latency: consecutive ones go to different accumulators (the four 128-column tiles of
// Oᵀ; four partial sums of Sᵀ, added up by the softmax threads).
static constexpr int kChains = 4;
static constexpr float kLog2e = 1.4426950408889634f;

struct Params {
  const int* block_table;
  const int* token_seq;          // null: token t is row t of the block table
  const int* positions;
  const long long* slots;
  float* part_o;
  float* part_ml;
  int max_blocks, block_size, num_blocks, num_splits, window;
  float scale;
  MbLatent L;
  int* error_flag;
};

__host__ __device__ inline int n_atoms(const MbLatent& L) { return (L.pitch + 63) / 64; }
__host__ __device__ inline int n_mtiles(const MbLatent& L) { return (L.rank_p + 127) / 128; }
// an odd number of latent atoms still needs room for a whole pair
__host__ __device__ inline int room(const MbLatent& L) {
  const int a = n_atoms(L), b = 2 * n_mtiles(L);
  return a > b ? a : b;
}
static size_t smem_bytes(const MbLatent& L) { return static_cast<size_t>(room(L)) * kAtom + n_atoms(L) * kQAtom + 2 * kPBytes + 3072; }

// v[h] of 32 lanes reduced over the warp for every h at once: lane h ends with the result of h (31 exchanges)
template <bool MAX>
__device__ __forceinline__ float transpose_reduce(float (&v)[32]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
    for (int j = 0; j < o; ++j) {
      const bool up = (lane & o) != 0;
      const float send = up ? v[j] : v[j + o], keep = up ? v[j + o] : v[j];
      const float other = __shfl_xor_sync(0xffffffffu, send, o);
      v[j] = MAX ? fmaxf(keep, other) : keep + other;
    }
  }
  return v[0];
}
__device__ __forceinline__ bool mbar_test(uint64_t* bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred P;\n\t"
      "mbarrier.test_wait.parity.shared::cta.b64 P, [%1], %2;\n\t"
      "selp.b32 %0, 1, 0, P;\n\t}\n"
      : "=r"(ok)
      : "r"(smem_u32(bar)), "r"(parity)
      : "memory");
  return ok != 0;
}
// barrier of one softmax warpgroup
__device__ __forceinline__ void bar_group(int g) { asm volatile("bar.sync %0, 128;" ::"r"(1 + g) : "memory"); }
// the same barrier, telling every thread of the group whether any of them gave up: they leave a loop together or not at all
__device__ __forceinline__ bool bar_group_or(int g, bool v) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 p, %1, 0;\n\t"
      "bar.red.or.pred q, %2, 128, p;\n\t"
      "selp.b32 %0, 1, 0, q;\n\t}\n"
      : "=r"(r)
      : "r"(static_cast<uint32_t>(v)), "r"(1 + g)
      : "memory");
  return r != 0;
}

// grid (splits, head groups of 32, tokens), 320 threads
__global__ void __launch_bounds__(320, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tm_c, const __grid_constant__ CUtensorMap tm_q, Params p) {
  extern __shared__ __align__(1024) uint8_t smem[];
  const MbLatent L = p.L;
  const int atoms = n_atoms(L), mtiles = n_mtiles(L), groups = mtiles + (atoms > 2 * mtiles ? 1 : 0);
  uint8_t* s_c = smem;
  uint8_t* s_q = s_c + room(L) * kAtom;
  uint8_t* s_p = s_q + atoms * kQAtom;
  float* s_red = reinterpret_cast<float*>(s_p + 2 * kPBytes);  // [2][4][32] per-warp results
  float* s_m = s_red + 256;                                    // [2][4][32] a copy per warp: maxima, then rescale factors
  float* s_ml = s_m + 256;                                     // [2][32] each group's sums at the end
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_ml + 64);
  uint64_t* full = bars;               // [2][5]: stage, atom pair
  uint64_t* empty = bars + 10;         // [2][5]
  uint64_t* q_full = bars + 20;
  uint64_t* s_full = bars + 21;        // [2]
  uint64_t* p_ready = bars + 23;       // [2]
  uint64_t* pv_done = bars + 25;       // [2]
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + 27);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);
  pdl_wait();
  const long long t = blockIdx.z;
  const int split = blockIdx.x, h0 = blockIdx.y * HT;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.slots[t] < 0 ? -1 : p.positions[t];
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int k0 = lo / TK * TK;                                 // tiles start on pages' 64-row boundaries
  const int total = pos < 0 ? 0 : (pos - k0) / TK + 1;
  const int per = (total + p.num_splits - 1) / p.num_splits;
  const int first = split * per, n_tiles = min(per, total - first);
  float* ml = p.part_ml + ((t * L.heads + h0) * p.num_splits + split) * 2;
  if (n_tiles <= 0) {
    pdl_trigger();
    if (threadIdx.x < HT && h0 + threadIdx.x < L.heads) {
      ml[threadIdx.x * p.num_splits * 2] = -INFINITY;
      ml[threadIdx.x * p.num_splits * 2 + 1] = 0.f;
    }
    return;
  }
  if (smem_u32(smem) & 1023u) {
    if (threadIdx.x == 0) atomicExch(p.error_flag, 45);
    return;
  }
  if (threadIdx.x == 0) {
    for (int g = 0; g < 10; ++g) {
      mbar_init(&full[g], 1);
      mbar_init(&empty[g], 1);
    }
    mbar_init(q_full, 1);
    for (int st = 0; st < 2; ++st) {
      mbar_init(&s_full[st], 1);
      mbar_init(&p_ready[st], 4);
      mbar_init(&pv_done[st], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_ptr, kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // a kernel behind this one may need tensor memory too: it is let in only after every CTA here has its own
  pdl_trigger();
  const uint32_t tmem = *tmem_ptr, tmem_o = tmem + 2 * kChains * HT;

  if (warp == 0) {
    if (elect_one()) {
      const int* bt = p.block_table + static_cast<long long>(p.token_seq != nullptr ? p.token_seq[t] : t) * p.max_blocks;
      const int oob = p.num_blocks * p.block_size;             // a row past the pool: filled with zeros
      auto row_of = [&](int key) -> int {
        if (key > pos) return oob;
        const int blk = bt[key / p.block_size];
        return blk >= 0 && blk < p.num_blocks ? blk * p.block_size + key % p.block_size : oob;
      };
      mbar_expect_tx(q_full, atoms * kQAtom);
      for (int a = 0; a < atoms; ++a) tma_load_2d(s_q + a * kQAtom, &tm_q, q_full, a * 64, static_cast<int>(t) * L.heads + h0);
      bool ok = true;
      for (int i = 0; i < n_tiles && ok && !*abort_flag; ++i) {
        const int st = i & 1, row = row_of(k0 + (first + i) * TK);
        for (int g = 0; g < groups && ok; ++g) {
          const int a0 = 2 * g, a1 = g < mtiles ? min(2 * g + 2, atoms) : atoms;
          ok = mbar_wait(&empty[st * 5 + g], ((i >> 1) & 1) ^ 1);
          if (!ok) break;
          mbar_expect_tx(&full[st * 5 + g], (a1 - a0) * (kAtom / 2));
          for (int a = a0; a < a1; ++a) tma_load_2d(s_c + a * kAtom + st * (kAtom / 2), &tm_c, &full[st * 5 + g], a * 64, row);
        }
      }
      if (!ok) { *abort_flag = 1; atomicExch(p.error_flag, 41); }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t idesc_s = make_idesc_bf16(2 * TK, HT, 0, 0);    // Sᵀ = C (K-major) · Q (K-major), both stages' rows
      constexpr uint32_t idesc_o = make_idesc_bf16(128, HT, 1, 1);       // Oᵀ = Cᵀ (MN-major) · P (MN-major)
      const uint32_t c_addr = smem_u32(s_c), q_addr = smem_u32(s_q), p_addr = smem_u32(s_p);
      const int steps = L.pitch / 16;
      // Whichever product can go next goes: scores of tile i as soon as its rows are here (at most one tile ahead), P·C of a tile as
      // soon as its softmax is done.  Neither waits behind the other: a tile's rows are given back, and refilled, at once.
      auto loaded = [&](int i) -> bool {
        bool r = true;
        for (int g = 0; g < groups && r; ++g) r = mbar_test(&full[(i & 1) * 5 + g], (i >> 1) & 1);
        return r;
      };
      bool ok = mbar_wait(q_full, 0);
      int s_next = 0, pv_next = 0;
      unsigned long long t_idle = 0;
      for (uint32_t spins = 0; pv_next < n_tiles && ok && !*abort_flag;) {
        bool moved = false;
        // (the buffer of Sᵀ has been read: its group arrived on p_ready of tile i − 2 after that, and PV i − 2 waited for it)
        if (s_next < n_tiles && s_next <= pv_next + 1 && loaded(s_next)) {
          const int st = s_next & 1;
          tc_fence_after();
          for (int a = 0; a < atoms; ++a) {
            const uint64_t dc = make_smem_desc_sw128(c_addr + a * kAtom, 16, 1024), dq = make_smem_desc_sw128(q_addr + a * kQAtom, 16, 1024);
#pragma unroll
            for (int k = 0; k < 4; ++k)          // the start address is the descriptor's low field, in 16-byte units
              if (a * 4 + k < steps) umma_bf16(tmem + (st * kChains + k) * HT, dc + k * 2, dq + k * 2, idesc_s, a != 0);
          }
          umma_commit(&s_full[st]);
          for (int g = mtiles; g < groups; ++g) umma_commit(&empty[st * 5 + g]);    // atoms without latent columns are done with
          ++s_next;
          moved = true;
        }
        if (pv_next < s_next && mbar_test(&p_ready[pv_next & 1], (pv_next >> 1) & 1)) {
          const int st = pv_next & 1;
          tc_fence_after();
          for (int m = 0; m < mtiles; ++m) {
#pragma unroll
            for (int part = 0; part < 2; ++part)
#pragma unroll
              for (int ks = 0; ks < TK / 16; ++ks)
                umma_bf16(tmem_o + st * 128 + m * HT,
                          make_smem_desc_sw128(c_addr + 2 * m * kAtom + st * (kAtom / 2) + ks * (16 * 128), kAtom, 1024),
                          make_smem_desc_sw128(p_addr + st * kPBytes + part * 64 + ks * (16 * 128), kPBytes, 1024), idesc_o,
                          ((pv_next >> 1) | part | ks) != 0);
            umma_commit(&empty[st * 5 + m]);
          }
          umma_commit(&pv_done[st]);
          ++pv_next;
          moved = true;
        }
        if (moved) {
          spins = 0;
          t_idle = 0;
        } else if ((++spins & 1023u) == 0) {
          const unsigned long long now = global_timer_ns();
          if (t_idle == 0) t_idle = now;
          else if (now - t_idle > kWaitLimitNs) ok = false;
        }
      }
      if (!ok) { *abort_flag = 1; atomicExch(p.error_flag, 42); }
    }
  } else {
    const int wg = (warp - 2) >> 2;                            // stage this group works for
    const int q4 = warp & 3, row = q4 * 32 + lane;             // row of Sᵀ, later latent column of an M tile
    const bool mine = (row >> 6) == wg;                        // the row is a key of this stage
    const uint32_t lane_off = static_cast<uint32_t>(q4 * 32) << 16;
    const uint32_t t_s = tmem + wg * kChains * HT + lane_off, t_o = tmem_o + wg * 128 + lane_off;
    const float sl2 = p.scale * kLog2e;
    float* red = s_red + wg * 128;
    float* my_m = s_m + wg * 128 + q4 * 32;
    float m_run = -INFINITY;                                   // reference maximum of head `lane` (all four warps the same)
    float l[32];
#pragma unroll
    for (int h = 0; h < 32; ++h) l[h] = 0.f;
    uint8_t* prow = s_p + wg * kPBytes + (row & 63) * 128;
    bool bad = false;                          // a wait ran out: go through the barriers with the others and leave behind the last one
    const int n_mine = (n_tiles + 1 - wg) / 2;
    for (int i = 0; i < n_mine; ++i) {
      bad = !mbar_wait(&s_full[wg], i & 1);
      tc_fence_after();
      float sum[32];
#pragma unroll
      for (int c = 0; c < kChains; ++c) {
        if (c < min(kChains, L.pitch / 16)) {
          uint32_t raw[32];
          tmem_ld_32x32(t_s + c * HT, raw);
          tmem_ld_wait();
#pragma unroll
          for (int h = 0; h < 32; ++h) sum[h] = c == 0 ? __uint_as_float(raw[h]) : sum[h] + __uint_as_float(raw[h]);
        }
      }
      const int key = k0 + (first + 2 * i + wg) * TK + (row & 63);
      const bool seen = mine && key >= lo && key <= pos;
      float s[32], v[32];
#pragma unroll
      for (int h = 0; h < 32; ++h) {
        s[h] = seen ? sum[h] * sl2 : -INFINITY;
        v[h] = s[h];
      }
      if (mine) red[q4 * 32 + lane] = transpose_reduce<true>(v);          // (a warp's rows all belong to one stage)
      bar_group(wg);
      float mx = fmaxf(m_run, fmaxf(red[wg * 64 + lane], red[wg * 64 + 32 + lane]));
      if (m_run != -INFINITY && mx - m_run <= 8.f) mx = m_run;            // lazy rescaling (see attention_tc.cu)
      const float alpha = m_run == -INFINITY ? 0.f : exp2f(m_run - mx);
      const bool moved = __any_sync(0xffffffffu, mx != m_run);            // the same in all four warps
      m_run = mx;
      // the previous product must be done before its P is overwritten and before Oᵀ is rescaled
      if (i > 0) {
        bad |= !mbar_wait(&pv_done[wg], (i - 1) & 1);
        tc_fence_after();
        if (moved) {
          my_m[lane] = alpha;
          __syncwarp();
#pragma unroll
          for (int h = 0; h < 32; ++h) l[h] *= my_m[h];
#pragma unroll 1
          for (int c = 0; c < mtiles; ++c) {
            uint32_t o[32];
            tmem_ld_32x32(t_o + c * HT, o);
            tmem_ld_wait();
#pragma unroll
            for (int h = 0; h < 32; ++h) o[h] = __float_as_uint(__uint_as_float(o[h]) * my_m[h]);
            tmem_st_32x32(t_o + c * HT, o);
          }
          tmem_st_wait();
          __syncwarp();
        }
      }
      if (mine) {
        my_m[lane] = m_run;
        __syncwarp();
#pragma unroll
        for (int c = 0; c < 4; ++c) {                                     // 8 heads: 16 bytes of P_hi and of P_lo
          float pv[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            pv[j] = exp2f(s[c * 8 + j] - my_m[c * 8 + j]);
            l[c * 8 + j] += pv[j];
          }
          uint32_t hi[4], lo4[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            hi[j] = pack_bf16x2(pv[2 * j], pv[2 * j + 1]);
            lo4[j] = pack_bf16x2(pv[2 * j] - __uint_as_float(hi[j] << 16), pv[2 * j + 1] - __uint_as_float(hi[j] & 0xffff0000u));
          }
          *reinterpret_cast<uint4*>(prow + ((c ^ (row & 7)) << 4)) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(prow + (((c + 4) ^ (row & 7)) << 4)) = make_uint4(lo4[0], lo4[1], lo4[2], lo4[3]);
        }
        fence_proxy_async();
      }
      tc_fence_before();
      bad = bar_group_or(wg, bad || *abort_flag);    // (red is read by everybody before the next tile writes it)
      if (bad) break;
      if (lane == 0) mbar_arrive(&p_ready[wg]);
    }
    if (!bad && n_mine > 0) bad = !mbar_wait(&pv_done[wg], (n_mine - 1) & 1);
    red[q4 * 32 + lane] = transpose_reduce<false>(l);
    if (bad) *abort_flag = 1;
    // both groups meet: maxima and sums of the other, and its Oᵀ through the shared memory of the tiles (all products are done)
    asm volatile("bar.sync 3, 256;" ::: "memory");
    if (__any_sync(0xffffffffu, *abort_flag)) {
      if (bad) atomicExch(p.error_flag, 43);
    } else {
      tc_fence_after();
      if (q4 == 0) {
        s_m[wg * 128 + lane] = m_run;
        s_ml[wg * 32 + lane] = (red[lane] + red[32 + lane]) + (red[64 + lane] + red[96 + lane]);
      }
      float* s_o = reinterpret_cast<float*>(s_c);              // [mtiles][32 heads][128 latent columns]
      if (wg == 1 && n_mine > 0)
#pragma unroll 1
        for (int m = 0; m < mtiles; ++m) {
          uint32_t o[32];
          tmem_ld_32x32(t_o + m * HT, o);
          tmem_ld_wait();
#pragma unroll
          for (int h = 0; h < 32; ++h) s_o[(m * 32 + h) * 128 + row] = __uint_as_float(o[h]);
        }
    }
    const bool stop = __any_sync(0xffffffffu, *abort_flag);
    asm volatile("bar.sync 3, 256;" ::: "memory");
    if (wg == 0 && !stop) {
      const float* s_o = reinterpret_cast<const float*>(s_c);
      const float m0 = s_m[lane], m1 = s_m[128 + lane], mm = fmaxf(m0, m1);
      const float f0 = exp2f(m0 - mm), f1 = m1 == -INFINITY ? 0.f : exp2f(m1 - mm);
      if (q4 == 0 && h0 + lane < L.heads) {
        ml[lane * p.num_splits * 2] = mm;
        ml[lane * p.num_splits * 2 + 1] = s_ml[lane] * f0 + s_ml[32 + lane] * f1;
      }
      const int n_h = min(HT, L.heads - h0);
      const bool both = n_tiles > 1;
#pragma unroll 1
      for (int m = 0; m < mtiles; ++m) {
        uint32_t a[32];
        tmem_ld_32x32(t_o + m * HT, a);
        tmem_ld_wait();
        const int c = m * 128 + row;
        float* dst = p.part_o + ((t * L.heads + h0) * p.num_splits + split) * L.rank_p + c;
#pragma unroll
        for (int h = 0; h < 32; ++h) {
          const float x0 = __shfl_sync(0xffffffffu, f0, h), x1 = __shfl_sync(0xffffffffu, f1, h);
          float r = __uint_as_float(a[h]) * x0;
          if (both) r = fmaf(s_o[(m * 32 + h) * 128 + row], x1, r);
          if (h < n_h && c < L.rank_p) dst[static_cast<long long>(h) * p.num_splits * L.rank_p] = r;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, kTmemCols);
  }
}

}  // namespace ldt
}  // namespace mb

using namespace mb;

// Splits of the keys of T tokens into part_o / part_ml (see mb_latent_decode).  block_size % 64 == 0, rank ≤ 512, pitch ≤ 640.
extern "C" int mb_latent_decode_tc(const void* q, const void* cache, const int* block_table, int max_blocks, int block_size,
                                   const int* token_seq, const int* positions, const long long* slots, float* part_o, float* part_ml, int T,
                                   float scale, int window, int splits, int num_blocks, MbLatent L, int* error_flag, cudaStream_t s) {
  if (block_size % 64 || L.rank_p > 512 || L.pitch > 640 || T > 65535) return -3;
  CUtensorMap tc, tq;
  int rc = make_tmap_bf16_2d(&tc, cache, static_cast<long long>(num_blocks) * block_size, L.pitch, L.pitch, 64, 64);
  if (rc) return 1000 + rc;
  rc = make_tmap_bf16_2d(&tq, q, static_cast<long long>(T) * L.heads, L.pitch, L.pitch, ldt::HT, 64);
  if (rc) return 2000 + rc;
  static bool once = false;
  if (!once) {
    const cudaError_t e = cudaFuncSetAttribute(ldt::latent_decode_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    once = true;
  }
  ldt::Params p{block_table, token_seq, positions, slots, part_o, part_ml, max_blocks, block_size, num_blocks, splits, window, scale, L, error_flag};
  return static_cast<int>(launch_pdl(ldt::latent_decode_tc_kernel, dim3(splits, (L.heads + ldt::HT - 1) / ldt::HT, T), dim3(320),
                                     ldt::smem_bytes(L), s, tc, tq, p));
}
