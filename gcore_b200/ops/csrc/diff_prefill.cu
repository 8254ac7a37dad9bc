// Prompt portions of differential attention on tcgen05, straight from the paged cache: two causal softmax maps over the same
// values per head, o = a1 - lambda * a2, normed over the head, scaled, gated.  A cached row is [2G keys | G values]; head h's
// maps read keys 2g and 2g + 1 and value g = h / (H / G).
//
// One CTA = 128 query rows of one head of one portion, both maps.  The portion's keys and those that earlier steps cached are
// read through the block table, tile by tile (64 keys, on 64-key boundaries of the sequence), by TMA; heads narrower than the
// tile are zero-filled by the loads.  A value tile serves both maps.  The probabilities feed the tensor core as two bf16 terms
// (rounded value, remainder), i.e. with 16 significant bits; they replace the scores in tensor memory (64 32-bit columns of S
// become 32 + 32 columns of packed pairs) and are the A operand of P V from there, so neither they nor their loads touch
// shared memory.  With M = 128 every TMEM lane is one query row.
//
//   warps 0-3, 4-7  softmax / O-correction of map 1, map 2 (thread t of a warpgroup <-> query row t <-> TMEM lane t); at the
//                   end both warpgroups read both accumulators, each for half of the columns, so the difference, its norm and
//                   the gate never leave the SM
//   warp 8          TMA producer (both queries once, then [key 1, key 2 | value] tiles into a ring)
//   warp 9          MMA issuer: both S_{j+1} are issued before P_j V_j, so score products overlap the softmax; they go to the
//                   buffer of P_{j-1} once its product is done
//
// TMEM columns (all 512, one CTA per SM): S and P of map m, buffer b at [64 (2m + b), +64); O of map m at [256 + m DV, +DV).
// Values wider than 128 columns take one CTA per 128 of them, which stores the difference for a finishing kernel.
#include "ptx.cuh"
#include "host_utils.h"
#include <float.h>

namespace gk {

constexpr int DF_BM = 128;
constexpr int DF_BN = 64;
constexpr int DF_THREADS = 320;
constexpr int DF_CHUNK = DF_BN * 128;   // one 64-column (128-byte) chunk of a key or value tile

struct DfParams {
  const int* tables;      // [portions, max_blocks]
  const int* cu;          // [portions + 1] first row of every portion
  const int* first_pos;   // [portions] tokens cached before the portion
  const __nv_bfloat16* gate;   // [rows, gate_ld]: a logit per head
  long long gate_ld;
  __nv_bfloat16* out;     // [rows, o_ld]: head h at h * vdim
  long long o_ld;
  const float* lam;
  float* partial;         // [rows, H, vdim] differences, when the values take more than one CTA; else null
  int H, G, vdim, true_vdim, max_blocks, num_blocks, block_size, vtiles;
  float scale, out_scale, eps;
  int* err;
};

// Two 32-bit numbers in a register pair: one instruction works on both.
__device__ __forceinline__ uint64_t pair2(float lo, float hi) {
  uint64_t v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(lo), "f"(hi));
  return v;
}
__device__ __forceinline__ float2 unpair2(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ float max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}

__device__ __forceinline__ void df_sync_softmax() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

template <int DQ, int DV>
struct DfGeo {
  static constexpr int NCH = DQ / 64, NCHV = DV / 64;
  static constexpr int STAGES = DQ == 64 ? 4 : 3;
  static constexpr int Q_BYTES = 2 * DF_BM * DQ * 2;
  static constexpr int K_BYTES = 2 * NCH * DF_CHUNK;
  static constexpr int V_BYTES = NCHV * DF_CHUNK;
  static constexpr int STAGE = K_BYTES + V_BYTES;
  static constexpr int BARS = Q_BYTES + STAGES * STAGE;
  static constexpr int SMEM = BARS + 256 + 2048;
  static_assert(SMEM <= 232448, "shared memory of one CTA");
};

template <int DQ, int DV>
__global__ void __launch_bounds__(DF_THREADS, 1)
diff_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                    const __grid_constant__ CUtensorMap tmV, DfParams p) {
  using Geo = DfGeo<DQ, DV>;
  constexpr int NCH = Geo::NCH, NCHV = Geo::NCHV, STAGES = Geo::STAGES;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* sQ = smem_raw;                                 // map, chunk
  uint8_t* sKV = sQ + Geo::Q_BYTES;                       // stage: key map, chunk | value chunk
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem_raw + Geo::BARS);
  uint64_t* q_full = bars;                                // 1
  uint64_t* k_full = q_full + 1;                          // STAGES
  uint64_t* v_full = k_full + STAGES;                     // STAGES
  uint64_t* kv_empty = v_full + STAGES;                   // STAGES
  uint64_t* s_full = kv_empty + STAGES;                   // map, buffer
  uint64_t* p_full = s_full + 4;                          // map, buffer (an arrival per warp): a map may be a tile ahead of the other
  uint64_t* pv_done = p_full + 4;                         // map, buffer
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(pv_done + 4);
  float* s_inv = reinterpret_cast<float*>(smem_raw + Geo::BARS + 256);   // map, row
  float* s_ss = s_inv + 256;

  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z / p.vtiles, v0 = (blockIdx.z % p.vtiles) * DV;
  const int r_beg = p.cu[b], len = p.cu[b + 1] - r_beg, p0 = p.first_pos[b];
  const int q0 = (gridDim.x - 1 - blockIdx.x) * DF_BM;    // the longest rows first
  if (q0 >= len) return;   // uniform across the CTA, before any allocation
  if (smem_u32(smem_raw) & 1023u) {
    if (threadIdx.x == 0) atomicCAS(p.err, 0, ERR_WAIT_MISC);
    return;
  }
  const int g = h / (p.H / p.G);
  const int last_row = q0 + DF_BM - 1 < len - 1 ? q0 + DF_BM - 1 : len - 1;
  const int last_key = p0 + last_row;                     // newest key any row of this CTA sees (absolute position)
  const int ntiles = last_key / DF_BN + 1;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < STAGES; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&kv_empty[i], 1);
    }
    for (int i = 0; i < 4; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[i], 4);
      mbar_init(&pv_done[i], 1);
    }
    fence_barrier_init();
    prefetch_tmap(&tmQ);
    prefetch_tmap(&tmK);
    prefetch_tmap(&tmV);
  }
  if (warp == 9) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t*>(tmem_holder);
  const uint32_t tmem_o = tmem_base + 4 * DF_BN;

  if (warp == 8) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      mbar_expect_tx(q_full, Geo::Q_BYTES);
#pragma unroll
      for (int i = 0; i < 2 * NCH; ++i)
        tma_load_3d(sQ + i * DF_BM * 128, &tmQ, q_full, (i % NCH) * 64, 2 * h + i / NCH, r_beg + q0);
    }
    __syncwarp();
    const int rows = p.block_size < DF_BN ? p.block_size : DF_BN;   // keys one load brings
    const int* table = p.tables + static_cast<long long>(b) * p.max_blocks;
    const int last_page = last_key / p.block_size;
    for (int it = 0; it < ntiles; ++it) {
      const int s = it % STAGES;
      if (!mbar_wait(&kv_empty[s], ((it / STAGES) & 1) ^ 1, p.err, ERR_WAIT_EMPTY)) break;
      if (lane == 0) {
        uint8_t* st = sKV + s * Geo::STAGE;
        mbar_expect_tx(&k_full[s], Geo::K_BYTES);
        mbar_expect_tx(&v_full[s], Geo::V_BYTES);
        for (int r = 0; r < DF_BN; r += rows) {
          // pages past the newest key are masked below: any valid page fills their rows
          int page = (it * DF_BN + r) / p.block_size;
          const int in_page = (it * DF_BN + r) % p.block_size;
          page = page < last_page ? page : last_page;
          int blk = table[page];
          blk = blk < 0 ? 0 : (blk >= p.num_blocks ? p.num_blocks - 1 : blk);
          const int at = blk * p.block_size + in_page;
#pragma unroll
          for (int i = 0; i < 2 * NCH; ++i)
            tma_load_3d(st + i * DF_CHUNK + r * 128, &tmK, &k_full[s], (i % NCH) * 64, 2 * g + i / NCH, at);
#pragma unroll
          for (int c = 0; c < NCHV; ++c)
            tma_load_3d(st + Geo::K_BYTES + c * DF_CHUNK + r * 128, &tmV, &v_full[s], v0 + c * 64, g, at);
        }
      }
      __syncwarp();
    }
  } else if (warp == 9) {
    // ------------------------------------------------------------------ MMA issuer
    constexpr uint32_t idesc_s = make_idesc(DF_BM, DF_BN, 1, 1, 0, 0);
    constexpr uint32_t idesc_o = make_idesc(DF_BM, DV, 1, 1, 0, 1);
    // descriptors of the first operands; the others are a distance away (the address is their lowest field, in 16-byte units)
    const uint64_t q_desc = make_smem_desc_sw128(smem_u32(sQ), 16, 1024), kv_desc = make_smem_desc_sw128(smem_u32(sKV), 16, 1024);
    const uint64_t v_desc = make_smem_desc_sw128(smem_u32(sKV + Geo::K_BYTES), DF_CHUNK, 1024);
    const bool leader = elect_one();
    bool ok = mbar_wait(q_full, 0, p.err, ERR_WAIT_FULL);
    auto issue_s = [&](int it) -> bool {
      const int s = it % STAGES, sb = it & 1;
      if (!mbar_wait(&k_full[s], (it / STAGES) & 1, p.err, ERR_WAIT_FULL)) return false;
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        if (it >= 2 && !mbar_wait(&pv_done[2 * m + sb], ((it - 2) >> 1) & 1, p.err, ERR_WAIT_TMEM_EMPTY)) return false;   // P of it - 2
        tc_fence_after();
        const uint64_t qd = q_desc + (m * NCH * DF_BM * 128 >> 4);
        const uint64_t kd = kv_desc + (s * Geo::STAGE + m * NCH * DF_CHUNK >> 4);
        if (leader) {
#pragma unroll
          for (int k4 = 0; k4 < DQ / 16; ++k4)
            umma_f16(tmem_base + (2 * m + sb) * DF_BN, qd + ((k4 >> 2) * DF_BM * 128 + (k4 & 3) * 32 >> 4),
                     kd + ((k4 >> 2) * DF_CHUNK + (k4 & 3) * 32 >> 4), idesc_s, k4 > 0 ? 1u : 0u);
          umma_commit(&s_full[2 * m + sb]);
        }
        __syncwarp();
      }
      return true;
    };
    if (ok) ok = issue_s(0);
    for (int it = 0; it < ntiles && ok; ++it) {
      const int s = it % STAGES;
      if (it + 1 < ntiles) {
        ok = issue_s(it + 1);
        if (!ok) break;
      }
      ok = mbar_wait(&v_full[s], (it / STAGES) & 1, p.err, ERR_WAIT_FULL);
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        if (ok) ok = mbar_wait(&p_full[2 * m + (it & 1)], (it >> 1) & 1, p.err, ERR_WAIT_MISC);
        if (!ok) break;
        tc_fence_after();
        const uint64_t vd = v_desc + (s * Geo::STAGE >> 4);
        const uint32_t pa = tmem_base + (2 * m + (it & 1)) * DF_BN;
        if (leader) {
#pragma unroll
          for (int term = 0; term < 2; ++term) {
#pragma unroll
            for (int k4 = 0; k4 < DF_BN / 16; ++k4)
              umma_f16_ts(tmem_o + m * DV, pa + term * 32 + k4 * 8, vd + (k4 * 2048 >> 4), idesc_o,
                          (it > 0 || term > 0 || k4 > 0) ? 1u : 0u);
          }
          if (m == 1) umma_commit(&kv_empty[s]);
          umma_commit(&pv_done[2 * m + (it & 1)]);
        }
        __syncwarp();
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax / correction / epilogue
    const int map = warp >> 2, row = threadIdx.x & 127;
    const int qi = q0 + row;               // row inside the portion
    const int pi = p0 + qi;                // its position in the sequence
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t my_o = tmem_o + map * DV + lane_addr;
    const float sl2 = p.scale * 1.4426950408889634f;
    float m = -FLT_MAX, l = 0.f;
    bool ok = true;
    for (int it = 0; it < ntiles; ++it) {
      const int sb = 2 * map + (it & 1);
      ok = mbar_wait(&s_full[sb], (it >> 1) & 1, p.err, ERR_WAIT_TMEM_FULL);
      if (!ok) break;
      tc_fence_after();
      float sv[DF_BN];
      {
        uint32_t r0[32], r1[32];         // both loads in flight
        tmem_ld32(tmem_base + lane_addr + sb * DF_BN, r0);
        tmem_ld32(tmem_base + lane_addr + sb * DF_BN + 32, r1);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          sv[j] = __uint_as_float(r0[j]);
          sv[32 + j] = __uint_as_float(r1[j]);
        }
      }
      const int kbase = it * DF_BN;
      if (kbase + DF_BN - 1 > pi) {
#pragma unroll
        for (int j = 0; j < DF_BN; ++j) sv[j] = kbase + j <= pi ? sv[j] : -FLT_MAX;
      }
      // four maxima at a time (chains are short), three operands an instruction
      float mx4[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) mx4[j] = max3(sv[3 * j], sv[3 * j + 1], sv[3 * j + 2]);
#pragma unroll
      for (int j = 12; j < DF_BN; j += 2) mx4[(j >> 1) & 3] = max3(mx4[(j >> 1) & 3], sv[j], sv[j + 1]);
      float mx = fmaxf(max3(mx4[0], mx4[1], mx4[2]), mx4[3]);
      if (mx != -FLT_MAX) mx *= sl2;       // log2 domain (the scale is positive)
      // the running maximum moves only when the tile exceeds it by more than 2^8, so the accumulator in tensor memory
      // is rescaled on few tiles; the probabilities then reach at most 256
      const float m_cand = fmaxf(m, mx);
      const bool grow = (m == -FLT_MAX) ? (m_cand != -FLT_MAX) : (m_cand > m + 8.f);
      const float m_new = grow ? m_cand : m;
      const float m_use = m_new == -FLT_MAX ? 0.f : m_new;
      const float corr = grow ? ex2(m - m_use) : 1.f;
      const uint64_t sl2x2 = pair2(sl2, sl2), m2 = pair2(-m_use, -m_use), minus1 = pair2(-1.f, -1.f);
      uint64_t ps[4] = {0, 0, 0, 0};
#pragma unroll
      for (int j = 0; j < DF_BN / 2; ++j) {
        const float2 x = unpair2(fma2(pair2(sv[2 * j], sv[2 * j + 1]), sl2x2, m2));
        sv[2 * j] = ex2(x.x);                            // masked scores underflow to exactly 0
        sv[2 * j + 1] = ex2(x.y);
        ps[j & 3] = add2(ps[j & 3], pair2(sv[2 * j], sv[2 * j + 1]));
      }
      const float2 sum = unpair2(add2(add2(ps[0], ps[1]), add2(ps[2], ps[3])));
      l = l * corr + (sum.x + sum.y);
      m = m_new;
      if (it > 0 && __any_sync(0xffffffff, grow)) {
        ok = mbar_wait(&pv_done[sb ^ 1], ((it - 1) >> 1) & 1, p.err, ERR_WAIT_MISC);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int c = 0; c < DV / 32; ++c) {
          uint32_t r[32];
          tmem_ld32(my_o + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * corr);
          tmem_st32(my_o + c * 32, r);
        }
      }
      // P over S: a column holds the keys 2j and 2j + 1; rounded values first, remainders behind
      uint32_t w[32];
#pragma unroll
      for (int j = 0; j < 32; ++j) w[j] = pack_bf16x2(sv[2 * j], sv[2 * j + 1]);
      tmem_st32(tmem_base + lane_addr + sb * DF_BN, w);
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        const float2 r = unpair2(fma2(pair2(__uint_as_float(w[j] << 16), __uint_as_float(w[j] & 0xffff0000u)), minus1,
                                      pair2(sv[2 * j], sv[2 * j + 1])));
        w[j] = pack_bf16x2(r.x, r.y);
      }
      tmem_st32(tmem_base + lane_addr + sb * DF_BN + 32, w);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[sb]);
    }
    // a buffer's barrier is at most one phase ahead or behind here: its product before this one was done when S was issued
    if (ok) ok = mbar_wait(&pv_done[2 * map + ((ntiles - 1) & 1)], ((ntiles - 1) >> 1) & 1, p.err, ERR_WAIT_MISC);
    // both accumulators are complete behind this barrier (every thread of both warpgroups arrives, whatever its waits did)
    s_inv[map * 128 + row] = l > 0.f ? 1.f / l : 0.f;
    tc_fence_before();
    df_sync_softmax();
    tc_fence_after();
    const float inv1 = s_inv[row], inv2 = s_inv[128 + row] * *p.lam;
    const int c0 = map * (DV / 2);         // this warpgroup's columns
    float d[DV / 2], ss = 0.f;
#pragma unroll
    for (int c = 0; c < DV / 64; ++c) {
      uint32_t r1[32], r2[32];
      tmem_ld32(tmem_o + lane_addr + c0 + c * 32, r1);
      tmem_ld32(tmem_o + lane_addr + DV + c0 + c * 32, r2);
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        const float v = __uint_as_float(r1[j]) * inv1 - __uint_as_float(r2[j]) * inv2;
        d[c * 32 + j] = v;
        ss = fmaf(v, v, ss);
      }
    }
    s_ss[map * 128 + row] = ss;
    df_sync_softmax();
    if (ok && qi < len) {
      const long long r = r_beg + qi;
      if (p.partial) {
        float* dst = p.partial + (r * p.H + h) * p.vdim + v0 + c0;
#pragma unroll
        for (int j = 0; j < DV / 2; j += 4)
          if (v0 + c0 + j < p.vdim) *reinterpret_cast<float4*>(dst + j) = make_float4(d[j], d[j + 1], d[j + 2], d[j + 3]);
      } else {
        const float gate = 1.f / (1.f + ex2(-1.4426950408889634f * __bfloat162float(p.gate[r * p.gate_ld + h])));
        const float f = p.out_scale * gate / sqrtf((s_ss[row] + s_ss[128 + row]) / p.true_vdim + p.eps);
        __nv_bfloat16* dst = p.out + r * p.o_ld + static_cast<long long>(h) * p.vdim + c0;
#pragma unroll
        for (int j = 0; j < DV / 2; j += 8) {
          if (c0 + j >= p.vdim) break;
          uint4 w;
          w.x = pack_bf16x2(d[j] * f, d[j + 1] * f);
          w.y = pack_bf16x2(d[j + 2] * f, d[j + 3] * f);
          w.z = pack_bf16x2(d[j + 4] * f, d[j + 5] * f);
          w.w = pack_bf16x2(d[j + 6] * f, d[j + 7] * f);
          *reinterpret_cast<uint4*>(dst + j) = w;
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

template <int DQ, int DV>
int launch_df(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const DfParams& p, dim3 grid,
              cudaStream_t st) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(diff_prefill_kernel<DQ, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         DfGeo<DQ, DV>::SMEM);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured = true;
  }
  launch_k(diff_prefill_kernel<DQ, DV>, grid, dim3(DF_THREADS), DfGeo<DQ, DV>::SMEM, st, tq, tk, tv, p);
  return launch_status();
}

}  // namespace gk

using namespace gk;

// 1 when a kernel is built for maps of `dim` and values of `vdim` columns
GK_EXPORT int gk_diff_prefill_supported(int dim, int vdim) { return dim >= 1 && dim <= 128 && vdim >= 1 && vdim <= 256; }

// q: the rotated queries of the packed projection (bf16, rows ld elements apart; head h's maps at (2h) * dim and
// (2h + 1) * dim); cache: rows of `row` elements, already with the portions' own keys (2G * dim columns) and values (at
// v_off).  block_size is 8, 16, 32 or a multiple of 64.  partial [rows, H, vdim]: needed for vdim > 128 only; it then
// receives the differences and `out` stays as it is.
// ptrs: {q, cache, tables, cu, first_pos, gate, out, lam, partial, err};  lds: {ld, gate_ld, o_ld, row}
// dims: {portions, rows, H, G, dim, vdim, true_vdim, v_off, block_size, max_blocks, max_portion, num_blocks}
// floats: {scale, out_scale, eps}
GK_EXPORT int gk_diff_prefill(void* const* ptrs, const long long* lds, const int* dims, const float* floats, void* stream) {
  const int n = dims[0], rows = dims[1], H = dims[2], G = dims[3], dim = dims[4], vdim = dims[5], bs = dims[8];
  const long long ld = lds[0], row = lds[3];
  if (!gk_diff_prefill_supported(dim, vdim) || G < 1 || H % G || dim % 8 || vdim % 8 || dims[7] % 8 || ld % 8 || row % 8 ||
      lds[2] % 8 || dims[6] < 1 || dims[6] > vdim || floats[0] <= 0.f)
    return -1;
  if (dims[7] < 2 * G * dim || row < dims[7] + G * vdim) return -1;
  if (bs < 8 || bs % 8 || (bs < DF_BN ? DF_BN % bs : bs % DF_BN)) return -2;
  if (n == 0) return 0;
  const __nv_bfloat16 *q = static_cast<const __nv_bfloat16*>(ptrs[0]), *cache = static_cast<const __nv_bfloat16*>(ptrs[1]);
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(ptrs[6])) & 15)
    return -1;
  if (vdim > 128 && !ptrs[8]) return -1;
  const int box = bs < DF_BN ? bs : DF_BN;
  const uint64_t tokens = static_cast<uint64_t>(dims[11]) * bs;
  CUtensorMap tq, tk, tv;
  if (make_tmap_3d(&tq, q, 2, rows, 2 * H, dim, ld, dim, DF_BM, 1, 64, true)) return -3;
  if (make_tmap_3d(&tk, cache, 2, tokens, 2 * G, dim, row, dim, box, 1, 64, true)) return -4;
  if (make_tmap_3d(&tv, cache + dims[7], 2, tokens, G, vdim, row, vdim, box, 1, 64, true)) return -5;
  DfParams p;
  p.tables = static_cast<const int*>(ptrs[2]); p.cu = static_cast<const int*>(ptrs[3]);
  p.first_pos = static_cast<const int*>(ptrs[4]);
  p.gate = static_cast<const __nv_bfloat16*>(ptrs[5]); p.gate_ld = lds[1];
  p.out = static_cast<__nv_bfloat16*>(ptrs[6]); p.o_ld = lds[2];
  p.lam = static_cast<const float*>(ptrs[7]);
  p.partial = vdim > 128 ? static_cast<float*>(ptrs[8]) : nullptr;
  p.err = static_cast<int*>(ptrs[9]);
  p.H = H; p.G = G; p.vdim = vdim; p.true_vdim = dims[6]; p.max_blocks = dims[9]; p.num_blocks = dims[11]; p.block_size = bs;
  p.vtiles = (vdim + 127) / 128;
  p.scale = floats[0]; p.out_scale = floats[1]; p.eps = floats[2];
  const dim3 grid((dims[10] + DF_BM - 1) / DF_BM, H, n * p.vtiles);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (dim <= 64) return vdim <= 64 ? launch_df<64, 64>(tq, tk, tv, p, grid, st) : launch_df<64, 128>(tq, tk, tv, p, grid, st);
  return vdim <= 64 ? launch_df<128, 64>(tq, tk, tv, p, grid, st) : launch_df<128, 128>(tq, tk, tv, p, grid, st);
}
