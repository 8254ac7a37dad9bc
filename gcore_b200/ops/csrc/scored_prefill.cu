// Prompt portions of grouped-query attention with a bias on every score, on tcgen05, straight from the paged cache (see
// scored_attention.cu for the mechanism and the layout of a cached row).  The weights are a softmax of
// (q . k) * scale - r1 ln(1 + r2 * distance) over a sliding window and the first `keep` positions, or (SIG)
// sigmoid((q . k) * scale + bias) over every earlier key, not normalised.
//
// One CTA = 256 query rows of one head of one portion, two tiles of 128 that share every key and value tile.  Keys are read
// through the block table, tile by tile (64 keys, on 64-key boundaries of the sequence), by TMA; heads narrower than the tile
// are zero-filled by the loads.  Tiles that hold kept positions come first, then those of the window; a query tile skips the
// tiles that none of its rows sees.  The weights feed the tensor core as two bf16 terms (rounded value, remainder), i.e. with
// 16 significant bits; they replace the scores in tensor memory (64 32-bit columns of S become 32 + 32 columns of packed pairs)
// and are the A operand of P V from there.  With M = 128 every TMEM lane is one query row.
//
//   warps 0-3, 4-7  weights / O-correction / epilogue of query tile 0, 1 (thread t of a warpgroup <-> row t <-> TMEM lane t)
//   warp 8          TMA producer (queries once, then [keys | values] tiles into a ring)
//   warp 9          MMA issuer: S_{j+1} of both query tiles is issued before P_j V_j, so score products overlap the weights
//
// The penalty depends on the distance alone: for a tile a warp computes the 95 values its 32 rows and 64 keys need, once each,
// into shared memory, where lane l reads consecutive words.  Two sigmoids share one reciprocal: 1/a = b / (a b).
//
// TMEM columns (all 512, one CTA per SM): S and P of query tile m, buffer b at [64 (2m + b), +64); O of m at [256 + m DV, +DV).
// Values wider than 128 columns take one CTA per 128 of them.
#include "ptx.cuh"
#include "host_utils.h"
#include <float.h>

namespace gk {

constexpr int SP_BM = 128;
constexpr int SP_BN = 64;
constexpr int SP_THREADS = 320;
constexpr int SP_CHUNK = SP_BN * 128;   // one 64-column (128-byte) chunk of a key or value tile
constexpr int SP_PEN = 96;              // penalties of a warp's tile

struct SpParams {
  const int* tables;      // [portions, max_blocks]
  const int* cu;          // [portions + 1] first row of every portion
  const int* first_pos;   // [portions] tokens cached before the portion
  const float *r1, *r2;   // [H] or null
  const float* head_bias; // SIG: [H] or null
  __nv_bfloat16* out;     // [rows, o_ld]: head h at h * vdim
  long long o_ld;
  int H, G, vdim, max_blocks, num_blocks, block_size, vtiles, window, keep;
  float scale, out_scale;
  int* err;
};

// Two 32-bit numbers in a register pair: one instruction works on both.
__device__ __forceinline__ uint64_t sp_pair(float lo, float hi) {
  uint64_t v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(lo), "f"(hi));
  return v;
}
__device__ __forceinline__ float2 sp_unpair(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ uint64_t sp_fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t sp_add2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ float sp_max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ float sp_rcp(float x) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
// A wait whose outcome is the same for the whole warp.
__device__ __forceinline__ bool sp_wait(uint64_t* bar, uint32_t phase, int* err, int code) {
  return __all_sync(0xffffffff, mbar_wait(bar, phase, err, code));
}

// The key tiles a CTA visits, and which of its two query tiles sees each.
struct SpTiles {
  int kept, first[2], last[2], count, keep;   // [first, last): tiles of the window; kept: leading tiles in front of it
  __device__ __forceinline__ SpTiles(int p0, int q0, int len, int window, int keep_) : keep(keep_) {
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const int q = q0 + m * SP_BM;
      first[m] = last[m] = 0;
      if (q >= len) continue;
      const int f = window > 0 ? p0 + q - window + 1 : 0;
      first[m] = f > 0 ? f / SP_BN : 0;
      last[m] = (p0 + (q + SP_BM - 1 < len - 1 ? q + SP_BM - 1 : len - 1)) / SP_BN + 1;
    }
    const int k = (keep + SP_BN - 1) / SP_BN;
    kept = k < first[0] ? k : first[0];
    const int end = last[1] > last[0] ? last[1] : last[0];
    count = kept + end - first[0];
  }
  __device__ __forceinline__ int tile(int it) const { return it < kept ? it : first[0] + it - kept; }
  __device__ __forceinline__ bool seen(int m, int t) const { return t < last[m] && (t >= first[m] || t * SP_BN < keep); }
};

template <int DQ, int DV>
struct SpGeo {
  static constexpr int NCH = DQ / 64, NCHV = DV / 64;
  static constexpr int STAGES = DQ == 64 ? 4 : 3;
  static constexpr int Q_BYTES = 2 * SP_BM * DQ * 2;
  static constexpr int K_BYTES = NCH * SP_CHUNK;
  static constexpr int V_BYTES = NCHV * SP_CHUNK;
  static constexpr int STAGE = K_BYTES + V_BYTES;
  static constexpr int BARS = Q_BYTES + STAGES * STAGE;
  static constexpr int PEN = BARS + 256;
  static constexpr int SMEM = PEN + 8 * SP_PEN * 4;
  static_assert(SMEM <= 232448, "shared memory of one CTA");
};

template <int DQ, int DV, bool SIG>
__global__ void __launch_bounds__(SP_THREADS, 1)
scored_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                      const __grid_constant__ CUtensorMap tmV, SpParams p) {
  using Geo = SpGeo<DQ, DV>;
  constexpr int NCH = Geo::NCH, NCHV = Geo::NCHV, STAGES = Geo::STAGES;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* sQ = smem_raw;                                 // query tile, chunk
  uint8_t* sKV = sQ + Geo::Q_BYTES;                       // stage: key chunk | value chunk
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem_raw + Geo::BARS);
  uint64_t* q_full = bars;                                // 1
  uint64_t* k_full = q_full + 1;                          // STAGES
  uint64_t* v_full = k_full + STAGES;                     // STAGES
  uint64_t* kv_empty = v_full + STAGES;                   // STAGES
  uint64_t* s_full = kv_empty + STAGES;                   // query tile, buffer
  uint64_t* p_full = s_full + 4;                          // query tile, buffer (an arrival per warp)
  uint64_t* pv_done = p_full + 4;                         // query tile, buffer
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(pv_done + 4);

  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z / p.vtiles, v0 = (blockIdx.z % p.vtiles) * DV;
  const int r_beg = p.cu[b], len = p.cu[b + 1] - r_beg, p0 = p.first_pos[b];
  const int q0 = (gridDim.x - 1 - blockIdx.x) * 2 * SP_BM;   // the longest rows first
  if (q0 >= len) return;   // uniform across the CTA, before any allocation
  if (smem_u32(smem_raw) & 1023u) {
    if (threadIdx.x == 0) atomicCAS(p.err, 0, ERR_WAIT_MISC);
    return;
  }
  const int g = h / (p.H / p.G);
  const SpTiles tiles(p0, q0, len, p.window, p.keep);

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
  const uint32_t tmem_o = tmem_base + 4 * SP_BN;

  if (warp == 8) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      mbar_expect_tx(q_full, Geo::Q_BYTES);
#pragma unroll
      for (int i = 0; i < 2 * NCH; ++i)
        tma_load_3d(sQ + i * SP_BM * 128, &tmQ, q_full, (i % NCH) * 64, h, r_beg + q0 + (i / NCH) * SP_BM);
    }
    __syncwarp();
    const int rows = p.block_size < SP_BN ? p.block_size : SP_BN;   // keys one load brings
    const int* table = p.tables + static_cast<long long>(b) * p.max_blocks;
    const int end = tiles.last[1] > tiles.last[0] ? tiles.last[1] : tiles.last[0];
    const int newest = p0 + (q0 + 2 * SP_BM - 1 < len - 1 ? q0 + 2 * SP_BM - 1 : len - 1);
    const int last_page = (newest < end * SP_BN - 1 ? newest : end * SP_BN - 1) / p.block_size;
    for (int it = 0; it < tiles.count; ++it) {
      const int s = it % STAGES;
      if (!sp_wait(&kv_empty[s], ((it / STAGES) & 1) ^ 1, p.err, ERR_WAIT_EMPTY)) break;
      if (lane == 0) {
        uint8_t* st = sKV + s * Geo::STAGE;
        mbar_expect_tx(&k_full[s], Geo::K_BYTES);
        mbar_expect_tx(&v_full[s], Geo::V_BYTES);
        const int key0 = tiles.tile(it) * SP_BN;
        for (int r = 0; r < SP_BN; r += rows) {
          // pages past the newest key are masked below: any valid page fills their rows
          int page = (key0 + r) / p.block_size;
          const int in_page = (key0 + r) % p.block_size;
          page = page < last_page ? page : last_page;
          int blk = table[page];
          blk = blk < 0 ? 0 : (blk >= p.num_blocks ? p.num_blocks - 1 : blk);
          const int at = blk * p.block_size + in_page;
#pragma unroll
          for (int c = 0; c < NCH; ++c) tma_load_3d(st + c * SP_CHUNK + r * 128, &tmK, &k_full[s], c * 64, g, at);
#pragma unroll
          for (int c = 0; c < NCHV; ++c)
            tma_load_3d(st + Geo::K_BYTES + c * SP_CHUNK + r * 128, &tmV, &v_full[s], v0 + c * 64, g, at);
        }
      }
      __syncwarp();
    }
  } else if (warp == 9) {
    // ------------------------------------------------------------------ MMA issuer
    constexpr uint32_t idesc_s = make_idesc(SP_BM, SP_BN, 1, 1, 0, 0);
    constexpr uint32_t idesc_o = make_idesc(SP_BM, DV, 1, 1, 0, 1);
    // descriptors of the first operands; the others are a distance away (the address is their lowest field, in 16-byte units)
    const uint64_t q_desc = make_smem_desc_sw128(smem_u32(sQ), 16, 1024), k_desc = make_smem_desc_sw128(smem_u32(sKV), 16, 1024);
    const uint64_t v_desc = make_smem_desc_sw128(smem_u32(sKV + Geo::K_BYTES), SP_CHUNK, 1024);
    const bool leader = elect_one();
    bool ok = sp_wait(q_full, 0, p.err, ERR_WAIT_FULL);
    int ns0 = 0, ns1 = 0, np0 = 0, np1 = 0;      // score and value products issued per query tile
    auto issue_s = [&](int it) -> bool {
      const int s = it % STAGES, t = tiles.tile(it);
      if (!sp_wait(&k_full[s], (it / STAGES) & 1, p.err, ERR_WAIT_FULL)) return false;
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        if (!tiles.seen(m, t)) continue;
        const int n = m ? ns1 : ns0, sb = n & 1;
        if (n >= 2 && !sp_wait(&pv_done[2 * m + sb], ((n - 2) >> 1) & 1, p.err, ERR_WAIT_TMEM_EMPTY)) return false;
        tc_fence_after();
        const uint64_t qd = q_desc + (m * NCH * SP_BM * 128 >> 4);
        const uint64_t kd = k_desc + (s * Geo::STAGE >> 4);
        if (leader) {
#pragma unroll
          for (int k4 = 0; k4 < DQ / 16; ++k4)
            umma_f16(tmem_base + (2 * m + sb) * SP_BN, qd + ((k4 >> 2) * SP_BM * 128 + (k4 & 3) * 32 >> 4),
                     kd + ((k4 >> 2) * SP_CHUNK + (k4 & 3) * 32 >> 4), idesc_s, k4 > 0 ? 1u : 0u);
          umma_commit(&s_full[2 * m + sb]);
        }
        __syncwarp();
        if (m) ++ns1;
        else ++ns0;
      }
      return true;
    };
    if (ok) ok = issue_s(0);
    for (int it = 0; it < tiles.count && ok; ++it) {
      const int s = it % STAGES, t = tiles.tile(it);
      if (it + 1 < tiles.count) {
        ok = issue_s(it + 1);
        if (!ok) break;
      }
      ok = sp_wait(&v_full[s], (it / STAGES) & 1, p.err, ERR_WAIT_FULL);
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        if (!tiles.seen(m, t)) continue;
        const int n = m ? np1 : np0, pb = 2 * m + (n & 1);
        if (ok) ok = sp_wait(&p_full[pb], (n >> 1) & 1, p.err, ERR_WAIT_MISC);
        if (!ok) break;
        tc_fence_after();
        const uint64_t vd = v_desc + (s * Geo::STAGE >> 4);
        const uint32_t pa = tmem_base + pb * SP_BN;
        if (leader) {
#pragma unroll
          for (int term = 0; term < 2; ++term) {
#pragma unroll
            for (int k4 = 0; k4 < SP_BN / 16; ++k4)
              umma_f16_ts(tmem_o + m * DV, pa + term * 32 + k4 * 8, vd + (k4 * 2048 >> 4), idesc_o,
                          (n > 0 || term > 0 || k4 > 0) ? 1u : 0u);
          }
          umma_commit(&pv_done[pb]);
        }
        __syncwarp();
        if (m) ++np1;
        else ++np0;
      }
      if (ok && leader) umma_commit(&kv_empty[s]);   // both products of the tile, and its scores long before
      __syncwarp();
    }
  } else {
    // ------------------------------------------------------------------ weights / correction / epilogue
    const int map = warp >> 2, row = threadIdx.x & 127;
    const int qi = q0 + map * SP_BM + row;   // row inside the portion
    const int pi = p0 + qi;                  // its position in the sequence
    const int lo = p.window > 0 ? pi - p.window + 1 : 0;
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t my_o = tmem_o + map * DV + lane_addr;
    const float sl2 = p.scale * 1.4426950408889634f;
    const float r1 = p.r1 ? -p.r1[h] : 0.f, r2 = p.r1 ? p.r2[h] : 0.f;
    const float bias = SIG && p.head_bias ? -1.4426950408889634f * p.head_bias[h] : 0.f;
    float* pen = reinterpret_cast<float*>(smem_raw + Geo::PEN) + warp * SP_PEN;
    float m = -FLT_MAX, l = 0.f;
    bool ok = true;
    int n = 0;                               // tiles this query tile has seen
    for (int it = 0; it < tiles.count; ++it) {
      const int t = tiles.tile(it);
      if (!tiles.seen(map, t)) continue;
      const int sb = 2 * map + (n & 1), kbase = t * SP_BN;
      if (!SIG) {
        // penalties of distances pi(lane 0) - kbase - 63 .. + 94; those below zero belong to masked keys
        const int d0 = pi - lane - kbase - (SP_BN - 1);
        __syncwarp();
#pragma unroll
        for (int k = 0; k < SP_PEN / 32; ++k) {
          const int d = d0 + lane + 32 * k;
          pen[lane + 32 * k] = r1 * __log2f(fmaf(r2, static_cast<float>(d > 0 ? d : 0), 1.f));
        }
        __syncwarp();
      }
      ok = sp_wait(&s_full[sb], (n >> 1) & 1, p.err, ERR_WAIT_TMEM_FULL);
      if (!ok) break;
      tc_fence_after();
      float sv[SP_BN];
      {
        uint32_t r0[32], r1_[32];          // both loads in flight
        tmem_ld32(tmem_base + lane_addr + sb * SP_BN, r0);
        tmem_ld32(tmem_base + lane_addr + sb * SP_BN + 32, r1_);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          sv[j] = __uint_as_float(r0[j]);
          sv[32 + j] = __uint_as_float(r1_[j]);
        }
      }
      const bool whole = kbase + SP_BN - 1 <= pi && (kbase >= lo || kbase + SP_BN <= p.keep);
      const bool all_whole = __all_sync(0xffffffff, whole);
      if (SIG) {
        const uint64_t nsl2 = sp_pair(-sl2, -sl2), b2 = sp_pair(bias, bias), one = sp_pair(1.f, 1.f);
#pragma unroll
        for (int j = 0; j < SP_BN / 2; ++j) {
          const float2 z = sp_unpair(sp_fma2(sp_pair(sv[2 * j], sv[2 * j + 1]), nsl2, b2));
          const float2 a = sp_unpair(sp_add2(sp_pair(ex2(fminf(z.x, 62.f)), ex2(fminf(z.y, 62.f))), one));
          const float r = sp_rcp(a.x * a.y);
          sv[2 * j] = r * a.y;
          sv[2 * j + 1] = r * a.x;
        }
        if (!all_whole) {
#pragma unroll
          for (int j = 0; j < SP_BN; ++j) {
            const int kj = kbase + j;
            sv[j] = kj <= pi && (kj >= lo || kj < p.keep) ? sv[j] : 0.f;
          }
        }
      } else {
        const float* pl = pen + lane + SP_BN - 1;
#pragma unroll
        for (int j = 0; j < SP_BN; ++j) sv[j] = fmaf(sv[j], sl2, pl[-j]);
        if (!all_whole) {
#pragma unroll
          for (int j = 0; j < SP_BN; ++j) {
            const int kj = kbase + j;
            sv[j] = kj <= pi && (kj >= lo || kj < p.keep) ? sv[j] : -FLT_MAX;
          }
        }
        // four maxima at a time (chains are short), three operands an instruction
        float mx4[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) mx4[j] = sp_max3(sv[3 * j], sv[3 * j + 1], sv[3 * j + 2]);
#pragma unroll
        for (int j = 12; j < SP_BN; j += 2) mx4[(j >> 1) & 3] = sp_max3(mx4[(j >> 1) & 3], sv[j], sv[j + 1]);
        const float mx = fmaxf(sp_max3(mx4[0], mx4[1], mx4[2]), mx4[3]);
        // the running maximum moves only when the tile exceeds it by more than 2^8, so the accumulator in tensor memory
        // is rescaled on few tiles; the weights then reach at most 256
        const float m_cand = fmaxf(m, mx);
        const bool grow = (m == -FLT_MAX) ? (m_cand != -FLT_MAX) : (m_cand > m + 8.f);
        const float m_new = grow ? m_cand : m;
        const float m_use = m_new == -FLT_MAX ? 0.f : m_new;
        const float corr = grow ? ex2(m - m_use) : 1.f;
        const uint64_t m2 = sp_pair(-m_use, -m_use);
        uint64_t ps[4] = {0, 0, 0, 0};
#pragma unroll
        for (int j = 0; j < SP_BN / 2; ++j) {
          const float2 x = sp_unpair(sp_add2(sp_pair(sv[2 * j], sv[2 * j + 1]), m2));
          sv[2 * j] = ex2(x.x);                            // masked scores underflow to exactly 0
          sv[2 * j + 1] = ex2(x.y);
          ps[j & 3] = sp_add2(ps[j & 3], sp_pair(sv[2 * j], sv[2 * j + 1]));
        }
        const float2 sum = sp_unpair(sp_add2(sp_add2(ps[0], ps[1]), sp_add2(ps[2], ps[3])));
        l = l * corr + (sum.x + sum.y);
        m = m_new;
        if (n > 0 && __any_sync(0xffffffff, grow)) {
          ok = sp_wait(&pv_done[sb ^ 1], ((n - 1) >> 1) & 1, p.err, ERR_WAIT_MISC);
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
      }
      // P over S: a column holds the keys 2j and 2j + 1; rounded values first, remainders behind
      const uint64_t minus1 = sp_pair(-1.f, -1.f);
      uint32_t w[32];
#pragma unroll
      for (int j = 0; j < 32; ++j) w[j] = pack_bf16x2(sv[2 * j], sv[2 * j + 1]);
      tmem_st32(tmem_base + lane_addr + sb * SP_BN, w);
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        const float2 r = sp_unpair(sp_fma2(sp_pair(__uint_as_float(w[j] << 16), __uint_as_float(w[j] & 0xffff0000u)), minus1,
                                           sp_pair(sv[2 * j], sv[2 * j + 1])));
        w[j] = pack_bf16x2(r.x, r.y);
      }
      tmem_st32(tmem_base + lane_addr + sb * SP_BN + 32, w);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[sb]);
      ++n;
    }
    // a buffer's barrier is at most one phase ahead or behind here: its product before this one was done when S was issued
    if (ok && n > 0) ok = sp_wait(&pv_done[2 * map + ((n - 1) & 1)], ((n - 1) >> 1) & 1, p.err, ERR_WAIT_MISC);
    tc_fence_after();
    if (ok && n > 0) {
      const float f = SIG ? p.out_scale : l > 0.f ? p.out_scale / l : 0.f;
      __nv_bfloat16* dst = p.out + static_cast<long long>(r_beg + qi) * p.o_ld + static_cast<long long>(h) * p.vdim + v0;
      const int cols = p.vdim - v0 < DV ? p.vdim - v0 : DV;
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t r[32];
        tmem_ld32(my_o + c * 32, r);
        tmem_ld_wait();
        if (qi < len) {
#pragma unroll
          for (int j = 0; j < 32; j += 8) {
            if (c * 32 + j >= cols) break;
            uint4 w;
            w.x = pack_bf16x2(__uint_as_float(r[j]) * f, __uint_as_float(r[j + 1]) * f);
            w.y = pack_bf16x2(__uint_as_float(r[j + 2]) * f, __uint_as_float(r[j + 3]) * f);
            w.z = pack_bf16x2(__uint_as_float(r[j + 4]) * f, __uint_as_float(r[j + 5]) * f);
            w.w = pack_bf16x2(__uint_as_float(r[j + 6]) * f, __uint_as_float(r[j + 7]) * f);
            *reinterpret_cast<uint4*>(dst + c * 32 + j) = w;
          }
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

template <int DQ, int DV, bool SIG>
int launch_sp(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const SpParams& p, dim3 grid,
              cudaStream_t st) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(scored_prefill_kernel<DQ, DV, SIG>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         SpGeo<DQ, DV>::SMEM);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured = true;
  }
  launch_k(scored_prefill_kernel<DQ, DV, SIG>, grid, dim3(SP_THREADS), SpGeo<DQ, DV>::SMEM, st, tq, tk, tv, p);
  return launch_status();
}

template <bool SIG>
int launch_sp_size(int dim, int vdim, const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const SpParams& p,
                   dim3 grid, cudaStream_t st) {
  if (dim <= 64)
    return vdim <= 64 ? launch_sp<64, 64, SIG>(tq, tk, tv, p, grid, st) : launch_sp<64, 128, SIG>(tq, tk, tv, p, grid, st);
  return vdim <= 64 ? launch_sp<128, 64, SIG>(tq, tk, tv, p, grid, st) : launch_sp<128, 128, SIG>(tq, tk, tv, p, grid, st);
}

}  // namespace gk

using namespace gk;

// 1 when a kernel is built for keys of `dim` and values of `vdim` columns
GK_EXPORT int gk_scored_prefill_supported(int dim, int vdim) { return dim >= 1 && dim <= 128 && vdim >= 1 && vdim <= 1024; }

// q: the prepared queries of the packed projection (bf16, rows ld elements apart; head h at h * dim); cache: rows of `row`
// elements, already with the portions' own keys (G * dim columns) and values behind them.  block_size is 8, 16, 32 or a
// multiple of 64.  sigmoid: sigmoids in place of the softmax;  window 0: unlimited.
// ptrs: {q, cache, tables, cu, first_pos, r1, r2, head_bias, out, err};  lds: {ld, o_ld, row}
// dims: {portions, rows, H, G, dim, vdim, block_size, max_blocks, max_portion, num_blocks, window, keep, sigmoid}
// floats: {scale, out_scale}
GK_EXPORT int gk_scored_prefill(void* const* ptrs, const long long* lds, const int* dims, const float* floats, void* stream) {
  const int n = dims[0], rows = dims[1], H = dims[2], G = dims[3], dim = dims[4], vdim = dims[5], bs = dims[6];
  const long long ld = lds[0], row = lds[2];
  if (!gk_scored_prefill_supported(dim, vdim) || G < 1 || H % G || dim % 8 || vdim % 8 || ld % 8 || row % 8 || lds[1] % 8)
    return -1;
  if (row < static_cast<long long>(G) * (dim + vdim) || dims[10] < 0 || dims[11] < 0) return -1;
  if ((ptrs[5] != nullptr) != (ptrs[6] != nullptr) || (dims[12] ? ptrs[5] != nullptr : ptrs[7] != nullptr)) return -1;
  if (bs < 8 || bs % 8 || (bs < SP_BN ? SP_BN % bs : bs % SP_BN)) return -2;
  if (n == 0) return 0;
  const __nv_bfloat16 *q = static_cast<const __nv_bfloat16*>(ptrs[0]), *cache = static_cast<const __nv_bfloat16*>(ptrs[1]);
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(ptrs[8])) & 15)
    return -1;
  const int box = bs < SP_BN ? bs : SP_BN;
  const uint64_t tokens = static_cast<uint64_t>(dims[9]) * bs;
  CUtensorMap tq, tk, tv;
  if (make_tmap_3d(&tq, q, 2, rows, H, dim, ld, dim, SP_BM, 1, 64, true)) return -3;
  if (make_tmap_3d(&tk, cache, 2, tokens, G, dim, row, dim, box, 1, 64, true)) return -4;
  if (make_tmap_3d(&tv, cache + static_cast<long long>(G) * dim, 2, tokens, G, vdim, row, vdim, box, 1, 64, true)) return -5;
  SpParams p;
  p.tables = static_cast<const int*>(ptrs[2]); p.cu = static_cast<const int*>(ptrs[3]);
  p.first_pos = static_cast<const int*>(ptrs[4]);
  p.r1 = static_cast<const float*>(ptrs[5]); p.r2 = static_cast<const float*>(ptrs[6]);
  p.head_bias = static_cast<const float*>(ptrs[7]);
  p.out = static_cast<__nv_bfloat16*>(ptrs[8]); p.o_ld = lds[1];
  p.err = static_cast<int*>(ptrs[9]);
  p.H = H; p.G = G; p.vdim = vdim; p.max_blocks = dims[7]; p.num_blocks = dims[9]; p.block_size = bs;
  p.vtiles = (vdim + 127) / 128;
  p.window = dims[10]; p.keep = dims[11];
  p.scale = floats[0]; p.out_scale = floats[1];
  const dim3 grid((dims[8] + 2 * SP_BM - 1) / (2 * SP_BM), H, n * p.vtiles);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return dims[12] ? launch_sp_size<true>(dim, vdim, tq, tk, tv, p, grid, st)
                  : launch_sp_size<false>(dim, vdim, tq, tk, tv, p, grid, st);
}
