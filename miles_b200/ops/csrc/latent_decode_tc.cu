// Decode attention over cached latents on tcgen05 tensor cores (bf16, pages of a multiple of 64 tokens).
//
// One CTA = (key split, 32 heads, token).  The KEYS are the 128-row side of both products and the heads the narrow side, so 32 heads
// fill an instruction and no row is padding:
//     Sᵀ [128 keys, 32]      = C · Qᵀ        C: tile of cached rows (K-major), Q: absorbed queries of 32 heads
//     Oᵀ [128 latent, 64] += Cᵀ · [P_hi | P_lo]   per 128 latent columns; the same tile in shared memory, read MN-major
// The softmax weights are two bf16 parts side by side in the N dimension: the tile is read once for both, and the parts' results
// are added up at the end (16 bits of mantissa).  A tile is nine (for 512 + 64 columns) 64-column atoms of 128 rows, brought by TMA
// page by page; an atom pair is refilled as soon as its part of Oᵀ is done, while the rest of the tile is still in use.
//   warp 0      TMA        warp 1      MMA issue, TMEM owner
//   warps 2..5  thread = key (softmax) and = latent column (rescaling, result)
// Keys before the window, after the token or outside the sequence get weight 0; a page-table entry outside the pool reads as zeros.
#include "mixers.cuh"
#include "ptx.cuh"

namespace mb {

int make_tmap_bf16_2d(CUtensorMap* out, const void* base, long long rows, long long cols, long long ld, int box_rows, int box_cols);

namespace ldt {

static constexpr int TK = 128, HT = 32;
static constexpr int kAtom = TK * 128, kQAtom = HT * 128, kPBytes = TK * 128;      // bytes: 64 columns of a tile / of the queries; P
static constexpr uint32_t kTmemCols = 512;                                         // Sᵀ: 32 columns; Oᵀ: 4 × 64 from column 64
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
static size_t smem_bytes(const MbLatent& L) { return static_cast<size_t>(room(L)) * kAtom + n_atoms(L) * kQAtom + kPBytes + 2048; }

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
__device__ __forceinline__ void bar_softmax() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
// the same barrier, telling every softmax thread whether any of them gave up: they leave a loop together or not at all
__device__ __forceinline__ bool bar_softmax_or(bool v) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 p, %1, 0;\n\t"
      "bar.red.or.pred q, 1, 128, p;\n\t"
      "selp.b32 %0, 1, 0, q;\n\t}\n"
      : "=r"(r)
      : "r"(static_cast<uint32_t>(v))
      : "memory");
  return r != 0;
}

// grid (splits, head groups of 32, tokens), 192 threads
__global__ void __launch_bounds__(192, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tm_c, const __grid_constant__ CUtensorMap tm_q, Params p) {
  extern __shared__ __align__(1024) uint8_t smem[];
  const MbLatent L = p.L;
  const int atoms = n_atoms(L), mtiles = n_mtiles(L), groups = mtiles + (atoms > 2 * mtiles ? 1 : 0);
  uint8_t* s_c = smem;
  uint8_t* s_q = s_c + room(L) * kAtom;
  uint8_t* s_p = s_q + atoms * kQAtom;
  float* s_red = reinterpret_cast<float*>(s_p + kPBytes);      // [4][32] per-warp results
  float* s_m = s_red + 128;                                    // [4][32] a copy per warp: maxima, then rescale factors
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_m + 128);
  uint64_t* full = bars;               // 6: per atom pair
  uint64_t* empty = bars + 6;          // 6
  uint64_t* q_full = bars + 12;
  uint64_t* s_full = bars + 13;
  uint64_t* p_ready = bars + 14;
  uint64_t* pv_done = bars + 15;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + 16);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_ptr + 1);
  pdl_wait();
  const long long t = blockIdx.z;
  const int split = blockIdx.x, h0 = blockIdx.y * HT;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.slots[t] < 0 ? -1 : p.positions[t];
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int k0 = lo / 64 * 64;                                 // tiles start on pages' 64-row boundaries
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
    for (int g = 0; g < 6; ++g) {
      mbar_init(&full[g], 1);
      mbar_init(&empty[g], 1);
    }
    mbar_init(q_full, 1);
    mbar_init(s_full, 1);
    mbar_init(p_ready, 4);
    mbar_init(pv_done, 1);
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
  const uint32_t tmem = *tmem_ptr, tmem_o = tmem + 64;

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
        const int key = k0 + (first + i) * TK;
        const int r0 = row_of(key), r1 = row_of(key + 64);
        for (int g = 0; g < groups && ok; ++g) {
          const int a0 = 2 * g, a1 = g < mtiles ? min(2 * g + 2, atoms) : atoms;
          ok = mbar_wait(&empty[g], (i & 1) ^ 1);
          if (!ok) break;
          mbar_expect_tx(&full[g], (a1 - a0) * kAtom);
          for (int a = a0; a < a1; ++a) {
            tma_load_2d(s_c + a * kAtom, &tm_c, &full[g], a * 64, r0);
            tma_load_2d(s_c + a * kAtom + kAtom / 2, &tm_c, &full[g], a * 64, r1);
          }
        }
      }
      if (!ok) { *abort_flag = 1; atomicExch(p.error_flag, 41); }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t idesc_s = make_idesc_bf16(TK, HT, 0, 0);        // Sᵀ = C (K-major) · Q (K-major)
      constexpr uint32_t idesc_o = make_idesc_bf16(128, 64, 1, 1);       // Oᵀ = Cᵀ (MN-major) · P (MN-major)
      const uint32_t c_addr = smem_u32(s_c), q_addr = smem_u32(s_q), p_addr = smem_u32(s_p);
      const int steps = L.pitch / 16;
      bool ok = mbar_wait(q_full, 0);
      for (int i = 0; i < n_tiles && ok && !*abort_flag; ++i) {
        // (the softmax threads have read the previous Sᵀ: they arrived on p_ready after that, and it was waited for)
        for (int ks = 0; ks < steps; ++ks) {
          if (ks % 8 == 0 && ks / 8 < groups) {
            ok = mbar_wait(&full[ks / 8], i & 1);
            if (!ok) break;
            tc_fence_after();
          }
          umma_bf16(tmem, make_smem_desc_sw128(c_addr + (ks >> 2) * kAtom + (ks & 3) * 32, 16, 1024),
                    make_smem_desc_sw128(q_addr + (ks >> 2) * kQAtom + (ks & 3) * 32, 16, 1024), idesc_s, ks != 0);
        }
        if (!ok) break;
        umma_commit(s_full);
        for (int g = mtiles; g < groups; ++g) umma_commit(&empty[g]);    // atoms without latent columns are done with
        ok = mbar_wait(p_ready, i & 1);
        if (!ok) break;
        tc_fence_after();
        for (int m = 0; m < mtiles; ++m) {
          for (int ks = 0; ks < TK / 16; ++ks)
            umma_bf16(tmem_o + m * 64, make_smem_desc_sw128(c_addr + 2 * m * kAtom + ks * (16 * 128), kAtom, 1024),
                      make_smem_desc_sw128(p_addr + ks * (16 * 128), kPBytes, 1024), idesc_o, (i | ks) != 0);
          umma_commit(&empty[m]);
        }
        umma_commit(pv_done);
      }
      if (!ok) { *abort_flag = 1; atomicExch(p.error_flag, 42); }
    }
  } else {
    const int q4 = warp & 3, row = q4 * 32 + lane;             // key of the tile, later latent column of an M tile
    const uint32_t lane_off = static_cast<uint32_t>(q4 * 32) << 16;
    const float sl2 = p.scale * kLog2e;
    float* my_m = s_m + q4 * 32;
    float m_run = -INFINITY;                                   // reference maximum of head `lane` (all four warps the same)
    float l[32];
#pragma unroll
    for (int h = 0; h < 32; ++h) l[h] = 0.f;
    uint8_t* prow = s_p + row * 128;
    bool bad = false;                          // a wait ran out: go through the barriers with the others and leave behind the last one
    for (int i = 0; i < n_tiles; ++i) {
      bad = !mbar_wait(s_full, i & 1);
      tc_fence_after();
      uint32_t raw[32];
      tmem_ld_32x32(tmem + lane_off, raw);
      tmem_ld_wait();
      const int key = k0 + (first + i) * TK + row;
      const bool seen = key >= lo && key <= pos;
      float s[32], v[32];
#pragma unroll
      for (int h = 0; h < 32; ++h) {
        s[h] = seen ? __uint_as_float(raw[h]) * sl2 : -INFINITY;
        v[h] = s[h];
      }
      s_red[q4 * 32 + lane] = transpose_reduce<true>(v);
      bar_softmax();
      float mx = m_run;
#pragma unroll
      for (int w = 0; w < 4; ++w) mx = fmaxf(mx, s_red[w * 32 + lane]);
      if (m_run != -INFINITY && mx - m_run <= 8.f) mx = m_run;            // lazy rescaling (see attention_tc.cu)
      const float alpha = m_run == -INFINITY ? 0.f : exp2f(m_run - mx);
      const bool moved = __any_sync(0xffffffffu, mx != m_run);            // the same in all four warps
      m_run = mx;
      // the previous product must be done before its P is overwritten and before Oᵀ is rescaled
      if (i > 0) {
        bad |= !mbar_wait(pv_done, (i - 1) & 1);
        tc_fence_after();
        if (moved) {
          my_m[lane] = alpha;
          __syncwarp();
#pragma unroll
          for (int h = 0; h < 32; ++h) l[h] *= my_m[h];
#pragma unroll 1
          for (int c = 0; c < mtiles * 2; ++c) {                          // columns c·32 + h belong to head h (hi and lo parts)
            uint32_t o[32];
            tmem_ld_32x32(tmem_o + lane_off + c * 32, o);
            tmem_ld_wait();
#pragma unroll
            for (int h = 0; h < 32; ++h) o[h] = __float_as_uint(__uint_as_float(o[h]) * my_m[h]);
            tmem_st_32x32(tmem_o + lane_off + c * 32, o);
          }
          tmem_st_wait();
          __syncwarp();
        }
      }
      my_m[lane] = m_run;
      __syncwarp();
#pragma unroll
      for (int c = 0; c < 4; ++c) {                                       // 8 heads: 16 bytes of P_hi and of P_lo
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
      tc_fence_before();
      bad = bar_softmax_or(bad || *abort_flag);      // (s_red is read by everybody before the next tile writes it)
      if (bad) break;
      if (lane == 0) mbar_arrive(p_ready);
    }
    if (!bad) bad = !mbar_wait(pv_done, (n_tiles - 1) & 1);
    bad = bar_softmax_or(bad);
    if (bad) {
      *abort_flag = 1;
      atomicExch(p.error_flag, 43);
    } else {
      tc_fence_after();
      s_red[q4 * 32 + lane] = transpose_reduce<false>(l);
      bar_softmax();
      if (q4 == 0 && h0 + lane < L.heads) {
        ml[lane * p.num_splits * 2] = m_run;
        ml[lane * p.num_splits * 2 + 1] = (s_red[lane] + s_red[32 + lane]) + (s_red[64 + lane] + s_red[96 + lane]);
      }
      const int n_h = min(HT, L.heads - h0);
#pragma unroll 1
      for (int m = 0; m < mtiles; ++m) {
        uint32_t a[32], b[32];
        tmem_ld_32x32(tmem_o + lane_off + m * 64, a);
        tmem_ld_32x32(tmem_o + lane_off + m * 64 + 32, b);
        tmem_ld_wait();
        const int c = m * 128 + row;
        if (c < L.rank_p) {
          float* dst = p.part_o + ((t * L.heads + h0) * p.num_splits + split) * L.rank_p + c;
#pragma unroll
          for (int h = 0; h < 32; ++h)
            if (h < n_h) dst[static_cast<long long>(h) * p.num_splits * L.rank_p] = __uint_as_float(a[h]) + __uint_as_float(b[h]);
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
  return static_cast<int>(launch_pdl(ldt::latent_decode_tc_kernel, dim3(splits, (L.heads + ldt::HT - 1) / ldt::HT, T), dim3(192),
                                     ldt::smem_bytes(L), s, tc, tq, p));
}
