// Prompt portions of sliding-window attention whose values are its keys, on tcgen05, straight from the paged cache:
// score = (q . k) * scale - slope_h * (i - j) over 0 <= i - j < window, softmax and probabilities in 32-bit.
//
// One CTA = 128 query rows of one head of one portion.  The portion's keys and those that earlier steps cached are read
// through the block table, tile by tile (64 keys, on 64-key boundaries of the sequence), by TMA; a tile is the B operand
// of S = Q K^T and, unchanged, the (MN-major) B operand of O += P K.  The probabilities feed the tensor core as two bf16
// terms (rounded value, remainder), i.e. with 16 significant bits.  With M = 128 every TMEM lane is one query row.
//
//   warps 0-3  softmax / O-correction / epilogue (thread t <-> query row t <-> TMEM lane t)
//   warp 4     TMA producer (Q once, then key tiles into a 3-stage ring)
//   warp 5     MMA issuer: S_{j+1} is issued before P_j K_j so the score product overlaps the softmax of the tile before
//
// TMEM columns (256 per CTA, two CTAs per SM): S buffers at [0, 64) and [64, 128), O at [128, 128 + D).
#include "ptx.cuh"
#include "host_utils.h"
#include <float.h>

namespace gk {

constexpr int WP_BM = 128;
constexpr int WP_BN = 64;
constexpr int WP_STAGES = 3;
constexpr int WP_THREADS = 192;

struct WpParams {
  const int* tables;      // [portions, max_blocks]
  const int* cu;          // [portions + 1] first row of every portion
  const int* first_pos;   // [portions] tokens cached before the portion
  const float* slopes;    // [H]
  __nv_bfloat16* out;     // [rows, H, D]
  int H, G, max_blocks, num_blocks, block_size, window;
  float scale;
  int* err;
};

template <int D>
__global__ void __launch_bounds__(WP_THREADS, 2)
window_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, WpParams p) {
  constexpr int NCH = D / 64;
  constexpr int Q_BYTES = WP_BM * D * 2;
  constexpr int K_BYTES = WP_BN * D * 2;
  constexpr int K_CHUNK = WP_BN * 128;
  constexpr int P_BYTES = WP_BM * WP_BN * 2;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* sQ = smem_raw;
  uint8_t* sK = sQ + Q_BYTES;
  uint8_t* sP = sK + WP_STAGES * K_BYTES;    // high terms, then remainders
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + 2 * P_BYTES);
  uint64_t* q_full = bars;                       // 1
  uint64_t* k_full = bars + 1;                   // WP_STAGES
  uint64_t* k_empty = k_full + WP_STAGES;        // WP_STAGES
  uint64_t* s_full = k_empty + WP_STAGES;        // 2
  uint64_t* s_empty = s_full + 2;                // 2 (128 arrivals)
  uint64_t* p_full = s_empty + 2;                // 1 (128 arrivals)
  uint64_t* pv_done = p_full + 1;                // 1
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(pv_done + 1);

  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z;
  const int r_beg = p.cu[b], len = p.cu[b + 1] - r_beg, p0 = p.first_pos[b];
  const int q0 = blockIdx.x * WP_BM;
  if (q0 >= len) return;   // uniform across the CTA, before any allocation
  if (smem_u32(smem_raw) & 1023u) {
    if (threadIdx.x == 0) atomicCAS(p.err, 0, ERR_WAIT_MISC);
    return;
  }
  const int g = h / (p.H / p.G);
  const int last_row = q0 + WP_BM - 1 < len - 1 ? q0 + WP_BM - 1 : len - 1;
  const int last_key = p0 + last_row;            // newest key any row of this CTA sees (absolute position)
  int first_key = p0 + q0 - p.window + 1;
  if (first_key < 0) first_key = 0;
  const int j_beg = first_key / WP_BN;
  const int ntiles = last_key / WP_BN + 1 - j_beg;   // >= 1

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < WP_STAGES; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&s_empty[i], 128);
    }
    mbar_init(p_full, 128);
    mbar_init(pv_done, 1);
    fence_barrier_init();
    prefetch_tmap(&tmQ);
    prefetch_tmap(&tmK);
  }
  if (warp == 5) {
    tmem_alloc(tmem_holder, 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t*>(tmem_holder);
  const uint32_t tmem_o = tmem_base + 2 * WP_BN;

  if (warp == 4) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      mbar_expect_tx(q_full, Q_BYTES);
#pragma unroll
      for (int c = 0; c < NCH; ++c) tma_load_3d(sQ + c * WP_BM * 128, &tmQ, q_full, c * 64, h, r_beg + q0);
    }
    __syncwarp();
    const int rows = p.block_size < WP_BN ? p.block_size : WP_BN;   // keys one load brings
    const int* table = p.tables + static_cast<long long>(b) * p.max_blocks;
    const int last_page = last_key / p.block_size;
    bool ok = true;
    for (int it = 0; it < ntiles; ++it) {
      const int s = it % WP_STAGES;
      ok = mbar_wait(&k_empty[s], ((it / WP_STAGES) & 1) ^ 1, p.err, ERR_WAIT_EMPTY);
      if (!ok) break;
      if (lane == 0) {
        mbar_expect_tx(&k_full[s], K_BYTES);
        const int key0 = (j_beg + it) * WP_BN;
        for (int r = 0; r < WP_BN; r += rows) {
          // pages past the newest key are masked below: any valid page fills their rows
          int page = (key0 + r) / p.block_size;
          const int in_page = (key0 + r) % p.block_size;
          page = page < last_page ? page : last_page;
          int blk = table[page];
          blk = blk < 0 ? 0 : (blk >= p.num_blocks ? p.num_blocks - 1 : blk);
#pragma unroll
          for (int c = 0; c < NCH; ++c)
            tma_load_3d(sK + s * K_BYTES + c * K_CHUNK + r * 128, &tmK, &k_full[s], c * 64, g,
                        blk * p.block_size + in_page);
        }
      }
      __syncwarp();
    }
  } else if (warp == 5) {
    // ------------------------------------------------------------------ MMA issuer
    constexpr uint32_t idesc_s = make_idesc(WP_BM, WP_BN, 1, 1, 0, 0);
    constexpr uint32_t idesc_o = make_idesc(WP_BM, D, 1, 1, 0, 1);
    bool ok = mbar_wait(q_full, 0, p.err, ERR_WAIT_FULL);
    auto issue_s = [&](int it) -> bool {
      const int s = it % WP_STAGES, sb = it & 1;
      if (!mbar_wait(&k_full[s], (it / WP_STAGES) & 1, p.err, ERR_WAIT_FULL)) return false;
      if (it >= 2 && !mbar_wait(&s_empty[sb], ((it - 2) >> 1) & 1, p.err, ERR_WAIT_TMEM_EMPTY)) return false;
      tc_fence_after();
      if (lane == 0) {
        const uint32_t qa = smem_u32(sQ), ka = smem_u32(sK + s * K_BYTES);
#pragma unroll
        for (int k4 = 0; k4 < D / 16; ++k4) {
          umma_f16(tmem_base + sb * WP_BN, make_smem_desc_sw128(qa + (k4 >> 2) * WP_BM * 128 + (k4 & 3) * 32, 16, 1024),
                   make_smem_desc_sw128(ka + (k4 >> 2) * K_CHUNK + (k4 & 3) * 32, 16, 1024), idesc_s, k4 > 0 ? 1u : 0u);
        }
        umma_commit(&s_full[sb]);
      }
      __syncwarp();
      return true;
    };
    if (ok) ok = issue_s(0);
    for (int it = 0; it < ntiles && ok; ++it) {
      const int s = it % WP_STAGES;
      if (it + 1 < ntiles) {
        ok = issue_s(it + 1);
        if (!ok) break;
      }
      ok = mbar_wait(p_full, it & 1, p.err, ERR_WAIT_MISC);
      if (!ok) break;
      tc_fence_after();
      if (lane == 0) {
        const uint32_t va = smem_u32(sK + s * K_BYTES);
#pragma unroll
        for (int term = 0; term < 2; ++term) {
          const uint32_t pa = smem_u32(sP + term * P_BYTES);
#pragma unroll
          for (int k4 = 0; k4 < WP_BN / 16; ++k4) {
            umma_f16(tmem_o, make_smem_desc_sw128(pa + k4 * 32, 16, 1024),
                     make_smem_desc_sw128(va + k4 * 2048, K_CHUNK, 1024), idesc_o,
                     (it > 0 || term > 0 || k4 > 0) ? 1u : 0u);
          }
        }
        umma_commit(&k_empty[s]);
        umma_commit(pv_done);
      }
      __syncwarp();
    }
  } else {
    // ------------------------------------------------------------------ softmax / correction / epilogue
    const int row = threadIdx.x;
    const int qi = q0 + row;               // row inside the portion
    const int pi = p0 + qi;                // its position in the sequence
    const uint32_t lane_addr = static_cast<uint32_t>(warp * 32) << 16;
    const float sl2 = p.scale * 1.4426950408889634f;
    const float slope2 = p.slopes[h] * 1.4426950408889634f;
    const int hi = pi;
    const int lo = pi - p.window + 1;
    float m = -FLT_MAX, l = 0.f;
    bool ok = true;
    for (int it = 0; it < ntiles; ++it) {
      const int sb = it & 1;
      ok = mbar_wait(&s_full[sb], (it >> 1) & 1, p.err, ERR_WAIT_TMEM_FULL);
      if (!ok) break;
      tc_fence_after();
      float sv[WP_BN];
#pragma unroll
      for (int c = 0; c < WP_BN / 32; ++c) {
        uint32_t r[32];
        tmem_ld32(tmem_base + lane_addr + sb * WP_BN + c * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) sv[c * 32 + j] = __uint_as_float(r[j]);
      }
      tc_fence_before();
      mbar_arrive(&s_empty[sb]);
      const int kbase = (j_beg + it) * WP_BN;
      // log2 domain: s * scale - slope * (pi - k)
      const float bias0 = -slope2 * static_cast<float>(pi - kbase);
      float mx = -FLT_MAX;
      if (kbase >= lo && kbase + WP_BN - 1 <= hi) {
#pragma unroll
        for (int j = 0; j < WP_BN; ++j) {
          sv[j] = fmaf(sv[j], sl2, fmaf(slope2, static_cast<float>(j), bias0));
          mx = fmaxf(mx, sv[j]);
        }
      } else {
#pragma unroll
        for (int j = 0; j < WP_BN; ++j) {
          const int kj = kbase + j;
          const float v = fmaf(sv[j], sl2, fmaf(slope2, static_cast<float>(j), bias0));
          sv[j] = (kj >= lo && kj <= hi) ? v : -FLT_MAX;
          mx = fmaxf(mx, sv[j]);
        }
      }
      // the running maximum moves only when the tile exceeds it by more than 2^8, so the accumulator in tensor memory
      // is rescaled on few tiles; the probabilities then reach at most 256
      const float m_cand = fmaxf(m, mx);
      const bool grow = (m == -FLT_MAX) ? (m_cand != -FLT_MAX) : (m_cand > m + 8.f);
      const float m_new = grow ? m_cand : m;
      const float m_use = m_new == -FLT_MAX ? 0.f : m_new;
      const float corr = grow ? ex2(m - m_use) : 1.f;
      float ps = 0.f;
#pragma unroll
      for (int j = 0; j < WP_BN; ++j) {
        const float e = ex2(sv[j] - m_use);   // masked scores underflow to exactly 0
        sv[j] = e;
        ps += e;
      }
      l = l * corr + ps;
      m = m_new;
      if (it > 0) {
        ok = mbar_wait(pv_done, (it - 1) & 1, p.err, ERR_WAIT_MISC);
        if (!ok) break;
        tc_fence_after();
        if (__any_sync(0xffffffff, grow)) {
#pragma unroll
          for (int c = 0; c < D / 32; ++c) {
            uint32_t r[32];
            tmem_ld32(tmem_o + lane_addr + c * 32, r);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * corr);
            tmem_st32(tmem_o + lane_addr + c * 32, r);
          }
          tmem_st_wait();
        }
      }
      // P -> shared, K-major with the 128-byte swizzle: 16-byte unit u of row r sits at unit u ^ (r & 7)
      uint8_t* rowp = sP + row * 128;
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        uint32_t w[4], v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float a = sv[u * 8 + 2 * e], c = sv[u * 8 + 2 * e + 1];
          w[e] = pack_bf16x2(a, c);
          const float ra = a - bf16_bits_to_float(static_cast<uint16_t>(w[e] & 0xffff));
          const float rc = c - bf16_bits_to_float(static_cast<uint16_t>(w[e] >> 16));
          v[e] = pack_bf16x2(ra, rc);
        }
        const int o = (u ^ (row & 7)) << 4;
        *reinterpret_cast<uint4*>(rowp + o) = make_uint4(w[0], w[1], w[2], w[3]);
        *reinterpret_cast<uint4*>(rowp + P_BYTES + o) = make_uint4(v[0], v[1], v[2], v[3]);
      }
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(p_full);
    }
    if (ok) {
      ok = mbar_wait(pv_done, (ntiles - 1) & 1, p.err, ERR_WAIT_MISC);
      if (ok) tc_fence_after();
    }
    if (ok) {
      const float inv = l > 0.f ? 1.f / l : 0.f;
      const bool valid = qi < len;
      __nv_bfloat16* orow = p.out + (static_cast<long long>(r_beg + qi) * p.H + h) * D;
#pragma unroll
      for (int c = 0; c < D / 32; ++c) {
        uint32_t r[32];
        tmem_ld32(tmem_o + lane_addr + c * 32, r);
        tmem_ld_wait();
        if (valid) {
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            uint4 w;
            w.x = pack_bf16x2(__uint_as_float(r[8 * j + 0]) * inv, __uint_as_float(r[8 * j + 1]) * inv);
            w.y = pack_bf16x2(__uint_as_float(r[8 * j + 2]) * inv, __uint_as_float(r[8 * j + 3]) * inv);
            w.z = pack_bf16x2(__uint_as_float(r[8 * j + 4]) * inv, __uint_as_float(r[8 * j + 5]) * inv);
            w.w = pack_bf16x2(__uint_as_float(r[8 * j + 6]) * inv, __uint_as_float(r[8 * j + 7]) * inv);
            *reinterpret_cast<uint4*>(orow + c * 32 + j * 8) = w;
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 256);
  }
}

template <int D>
int launch_wp(const CUtensorMap& tq, const CUtensorMap& tk, const WpParams& p, dim3 grid, cudaStream_t st) {
  constexpr int SMEM = WP_BM * D * 2 + WP_STAGES * WP_BN * D * 2 + 2 * WP_BM * WP_BN * 2 + 256;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(window_prefill_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    if (e != cudaSuccess) return static_cast<int>(e);
    cudaFuncSetAttribute(window_prefill_kernel<D>, cudaFuncAttributePreferredSharedMemoryCarveout,
                         cudaSharedmemCarveoutMaxShared);
    configured = true;
  }
  launch_k(window_prefill_kernel<D>, grid, dim3(WP_THREADS), SMEM, st, tq, tk, p);
  return launch_status();
}

}  // namespace gk

using namespace gk;

// proj: packed projection rows (bf16, `ld` elements apart) with the queries at column q_off; cache [num_blocks,
// block_size, G, D] already holds the portions' own keys.  block_size is 8, 16, 32 or a multiple of 64.
// dims: {portions, rows, H, G, D, window, block_size, max_blocks, max_portion, q_off, num_blocks, 0}
GK_EXPORT int gk_window_prefill(const void* proj, long long ld, const void* cache, const int* tables, const int* cu,
                                const int* first_pos, const float* slopes, void* out, const int* dims, float scale,
                                int* err, void* stream) {
  const int n = dims[0], rows = dims[1], H = dims[2], G = dims[3], D = dims[4], bs = dims[6];
  if ((D != 64 && D != 128) || H % G || dims[5] < 1 || ld % 8 || dims[9] % 8) return -1;
  if (bs < 8 || bs % 8 || (bs < WP_BN ? WP_BN % bs : bs % WP_BN)) return -2;
  if (n == 0) return 0;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(proj) + dims[9];
  if (reinterpret_cast<uintptr_t>(q) & 15) return -1;
  const int box_rows = bs < WP_BN ? bs : WP_BN;
  CUtensorMap tq, tk;
  if (make_tmap_3d(&tq, q, 2, rows, H, D, ld, D, WP_BM, 1, 64, true)) return -3;
  if (make_tmap_3d(&tk, cache, 2, static_cast<uint64_t>(dims[10]) * bs, G, D, static_cast<uint64_t>(G) * D, D, box_rows, 1,
                   64, true))
    return -4;
  WpParams p;
  p.tables = tables; p.cu = cu; p.first_pos = first_pos; p.slopes = slopes;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.H = H; p.G = G; p.max_blocks = dims[7]; p.num_blocks = dims[10]; p.block_size = bs; p.window = dims[5];
  p.scale = scale; p.err = err;
  const dim3 grid((dims[8] + WP_BM - 1) / WP_BM, H, n);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return D == 64 ? launch_wp<64>(tq, tk, p, grid, st) : launch_wp<128>(tq, tk, p, grid, st);
}
