// Grouped-query attention with a bias on every score, around the prompt kernel (scored_prefill.cu).  The weights of the keys are
// a softmax of the scores, from which r1 * ln(1 + r2 * distance) may be taken off, over a sliding window and the first `keep`
// positions; or sigmoids of score + a number per head, not normalised.  Queries and keys may be rotated and divided by their
// root mean square.  A cached row is [G keys | G values].
//   * head_prep_kernel      rows of a packed projection: queries rotated / normed in place, keys likewise into their cache slot
//                           (or in place), values to the slot;
//   * silu_columns_kernel   columns of a packed projection replaced by their silu;
//   * scored_decode_kernel  one new token per request, bf16, KV splits, on mma.sync tiles whose rows are the query heads of a
//                           group (far below the 64-row minimum of a tcgen05 instruction).  Rotation, norm and append of the new
//                           token are part of it;
//   * scored_merge_kernel   merges the KV splits.
// Weights stay 32-bit: for the tensor core they are split into two bf16 terms (rounded value, remainder).
#include "ptx.cuh"
#include "host_utils.h"
#include "rotary.cuh"
#include <cuda_bf16.h>
#include <float.h>
#include <type_traits>

namespace gk {

constexpr int SA_MAX_ROT = 512;
constexpr float SA_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float2 sa_ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 sa_ld2(const __nv_bfloat16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
__device__ __forceinline__ void sa_st2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void sa_st2(__nv_bfloat16* p, float2 v) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y);
}
__device__ __forceinline__ float2 sa_rotate(float2 v, float c, float s) {
  return make_float2(v.x * c - v.y * s, v.y * c + v.x * s);
}
__device__ __forceinline__ float sa_warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffff, v, o);
  return v;
}

template <typename T>
struct HeadPrepParams {
  T* proj;                 // packed projection rows
  long long ld;
  int q_off, k_off, v_off; // NQ queries, NK keys of D columns each, VC value columns
  int NQ, NK, D, VC, rot;  // rot leading dimensions are rotated, neighbours paired
  const float2* turns;     // [rot / 2] turns per position: value, remainder
  const int *pos, *slots;  // cache slot of every row; negative: not stored
  T* cache;                // rows of NK * D + VC, or null: keys in place, values left alone
  int true_D;              // dimensions the norm's mean is taken over; 0: no norm
  float eps;
};

// Eight elements at a time.
__device__ __forceinline__ void sa_ld8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void sa_ld8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    v[2 * i] = __uint_as_float(w[i] << 16);
    v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}
__device__ __forceinline__ void sa_st8(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void sa_st8(__nv_bfloat16* p, const float (&v)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]),
                                            pack_bf16x2(v[6], v[7]));
}

// One CTA per row; GL lanes (a power of two) per head, each with NU times eight neighbouring elements.
template <typename T, int GL, int NU>
__global__ void __launch_bounds__(128) head_prep_kernel(const HeadPrepParams<T> p) {
  __shared__ __align__(16) float s_cos[SA_MAX_ROT / 2], s_sin[SA_MAX_ROT / 2];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, tid = threadIdx.x, half = p.rot >> 1;
  T* pr = p.proj + row * p.ld;
  const int slot = p.slots ? p.slots[row] : -1;
  if (half) {
    const int pos = p.pos[row];
    for (int i = tid; i < half; i += 128) rotation_at(pos, p.turns[i], &s_sin[i], &s_cos[i]);
    __syncthreads();
  }
  T* dst_row = p.cache ? p.cache + static_cast<long long>(slot < 0 ? 0 : slot) * (p.NK * p.D + p.VC) : nullptr;
  const int heads = p.NQ + (p.cache && slot < 0 ? 0 : p.NK), gl = tid % GL;
  for (int h0 = 0; h0 < heads; h0 += 128 / GL) {            // the same number of rounds for every lane
    const int h = h0 + tid / GL;
    const bool key = h >= p.NQ;
    const int n = key ? h - p.NQ : h;
    T* src = pr + (key ? p.k_off : p.q_off) + static_cast<long long>(n) * p.D;
    T* dst = key && dst_row ? dst_row + n * p.D : src;
    float v[NU][8], ss = 0.f;
#pragma unroll
    for (int u = 0; u < NU; ++u) {
      const int d = (u * GL + gl) * 8;
#pragma unroll
      for (int e = 0; e < 8; ++e) v[u][e] = 0.f;
      if (h < heads && d < p.D) sa_ld8(src + d, v[u]);
#pragma unroll
      for (int e = 0; e < 8; e += 2) {
        if (d + e < p.rot) {
          const float2 r = sa_rotate(make_float2(v[u][e], v[u][e + 1]), s_cos[(d + e) >> 1], s_sin[(d + e) >> 1]);
          v[u][e] = r.x;
          v[u][e + 1] = r.y;
        }
        ss = fmaf(v[u][e], v[u][e], fmaf(v[u][e + 1], v[u][e + 1], ss));
      }
    }
    if (p.true_D) {
#pragma unroll
      for (int o = GL / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffff, ss, o);
      const float f = 1.f / sqrtf(ss / p.true_D + p.eps);
#pragma unroll
      for (int u = 0; u < NU; ++u) {
#pragma unroll
        for (int e = 0; e < 8; ++e) v[u][e] *= f;
      }
    }
#pragma unroll
    for (int u = 0; u < NU; ++u) {
      const int d = (u * GL + gl) * 8;
      if (h < heads && d < p.D) sa_st8(dst + d, v[u]);
    }
  }
  if (dst_row && slot >= 0)
    for (int c = tid * 8; c < p.VC; c += 128 * 8) {
      float v[8];
      sa_ld8(pr + p.v_off + c, v);
      sa_st8(dst_row + p.NK * p.D + c, v);
    }
}

template <typename T>
int launch_head_prep(const HeadPrepParams<T>& p, int rows, cudaStream_t st) {
  const dim3 grid(rows), block(128);
  if (p.D <= 32) launch_k(head_prep_kernel<T, 4, 1>, grid, block, 0, st, p);
  else if (p.D <= 64) launch_k(head_prep_kernel<T, 8, 1>, grid, block, 0, st, p);
  else if (p.D <= 128) launch_k(head_prep_kernel<T, 16, 1>, grid, block, 0, st, p);
  else if (p.D <= 256) launch_k(head_prep_kernel<T, 32, 1>, grid, block, 0, st, p);
  else if (p.D <= 1024) launch_k(head_prep_kernel<T, 32, 4>, grid, block, 0, st, p);
  else return -2;
  return launch_status();
}

// Eight columns a thread: x over the columns, rows blockIdx.y, + gridDim.y, ...
template <typename T>
__global__ void __launch_bounds__(256) silu_columns_kernel(T* __restrict__ proj, long long ld, int off, int n, int rows) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * 256 + threadIdx.x) * 8;
  if (c >= n) return;
  for (int r = blockIdx.y; r < rows; r += gridDim.y) {
    T* at = proj + r * ld + off + c;
    float v[8];
    sa_ld8(at, v);
#pragma unroll
    for (int e = 0; e < 8; ++e)
      v[e] = std::is_same<T, float>::value ? v[e] / (1.f + expf(-v[e])) : __fdividef(v[e], 1.f + __expf(-v[e]));
    sa_st8(at, v);
  }
}

// ---------------------------------------------------------------------------------------------------- bf16 decode
__device__ __forceinline__ void sa_ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sa_ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void sa_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float sa_rest(float v) { return v - __bfloat162float(__float2bfloat16(v)); }

constexpr int SDK_WARPS = 4;
constexpr int SDK_ROWS = 16;         // query heads per CTA (rows of an mma tile)
constexpr int SDK_MIN_SPLIT = 128;
constexpr int SDK_MAX_SPLITS = 256;
inline int& scored_decode_target_ctas() {
  static int n = 444;
  return n;
}

struct ScoredDecodeParams {
  const __nv_bfloat16* proj;   // packed rows, one per request, neither rotated nor normed yet
  long long ld;
  int q_off, k_off, v_off;
  __nv_bfloat16* cache;        // rows of `row` elements: G keys of `dim`, G values of `vdim` columns
  int row;
  const int* tables;
  int max_blocks, block_size;
  const int* ctx_len;          // counts the new token; 0: inactive
  const int* new_slots;
  const float2* turns;         // with rot
  const float *r1, *r2;        // distance penalty per head, or null
  const float* head_bias;      // SIG: [H] or null
  __nv_bfloat16* out;
  long long o_ld;
  float* scratch;              // [B, H, nsplit, vdim + 2]
  int H, G, dim, vdim, rot, true_dim, window, keep, nsplit, split_tokens;
  float scale, out_scale, eps;
};

// What a token at position len - 1 sees, as consecutive places: the kept positions outside the window first, then the window.
struct SeenKeys {
  int kept, start, count;
  __device__ __forceinline__ SeenKeys(int len, int window, int keep) {
    start = window > 0 && len > window ? len - window : 0;
    kept = keep < start ? keep : start;
    count = kept + len - start;
  }
  __device__ __forceinline__ int position(int place) const { return place < kept ? place : start + place - kept; }
};

// DP: columns of a key tile (dim <= DP), DV: of a value tile, TOK: tokens per warp tile.
template <int DP, int DV, int TOK>
struct SdGeo {
  static constexpr int RK = 2 * DP, RV = 2 * DV;                     // bytes of a key / value tile row
  static constexpr int WARP = TOK * (RK + RV);
  static constexpr int TILES = SDK_WARPS * WARP, MERGE = SDK_WARPS * SDK_ROWS * DV * 4;
  static constexpr int BODY = TILES > MERGE ? TILES : MERGE;
  static constexpr int SMEM = BODY + SDK_ROWS * RK;                  // the queries behind the tiles
  static constexpr int CTAS = SMEM <= 56 * 1024 && DV <= 128 ? 4 : SMEM <= 72 * 1024 && DV <= 128 ? 3 : 2;
};

// grid (request, kv head x blocks of 16 heads, split).  ONE8: groups of up to 8 heads; rows 8-15 of the probability tile then
// carry the remainder terms of rows 0-7, so one product serves both terms.  SIG: sigmoids in place of the softmax.
template <int DP, int DV, int TOK, bool ONE8, bool SIG>
__global__ void __launch_bounds__(SDK_WARPS * 32, (SdGeo<DP, DV, TOK>::CTAS)) scored_decode_kernel(const ScoredDecodeParams p) {
  using Geo = SdGeo<DP, DV, TOK>;
  constexpr int NT = TOK / 8;          // score tiles of 8 tokens
  constexpr int NO = DV / 8;           // output tiles of 8 columns
  constexpr int KS = DP / 16;          // k-steps
  constexpr int HV = ONE8 ? 1 : 2;     // row halves that hold scores
  extern __shared__ __align__(128) uint8_t sd_smem[];
  __shared__ float m_all[SDK_WARPS][SDK_ROWS], l_all[SDK_WARPS][SDK_ROWS];
  __shared__ float s_cos[DP / 2], s_sin[DP / 2];
  __shared__ __align__(16) __nv_bfloat16 s_key[DP];   // the new key, rotated and normed

  pdl_launch_dependents();
  pdl_wait();
  const int grp = p.H / p.G, hblocks = (grp + SDK_ROWS - 1) / SDK_ROWS;
  const int b = blockIdx.x, g = blockIdx.y / hblocks, hb = blockIdx.y % hblocks, split = blockIdx.z;
  const int h0 = g * grp + hb * SDK_ROWS;
  const int nh = grp - hb * SDK_ROWS < SDK_ROWS ? grp - hb * SDK_ROWS : SDK_ROWS;
  const int len = p.ctx_len[b];
  const SeenKeys seen(len, p.window, p.keep);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int s0 = split * p.split_tokens;
  if (split > 0 && s0 >= seen.count) return;                   // dead split: the merge kernel skips it
  const int s1 = s0 + p.split_tokens < seen.count ? s0 + p.split_tokens : seen.count;
  const int ntiles = s1 > s0 ? (s1 - s0 + TOK - 1) / TOK : 0;
  const __nv_bfloat16* prow = p.proj + b * p.ld;
  const int kc = p.dim >> 3, vc = p.vdim >> 3;                 // 16-byte chunks in use

  uint8_t* kt = sd_smem + warp * Geo::WARP;
  uint8_t* vt = kt + TOK * Geo::RK;
  uint8_t* sq = sd_smem + Geo::BODY;
  const uint32_t kts = static_cast<uint32_t>(__cvta_generic_to_shared(kt));
  const uint32_t vts = static_cast<uint32_t>(__cvta_generic_to_shared(vt));
  // chunk ch of row r: the low three chunk bits are xor-ed with the row, so an ldmatrix is free of bank conflicts
  auto at = [](int r, int ch, int row_bytes) { return r * row_bytes + (((ch & ~7) | ((ch ^ r) & 7)) << 4); };
  auto slot_of = [&](int t) -> int {
    const int place = s0 + t * TOK + (lane < TOK ? lane : TOK - 1);
    if (place >= s1) return -1;
    const int j = seen.position(place);
    return p.tables[static_cast<long long>(b) * p.max_blocks + j / p.block_size] * p.block_size + j % p.block_size;
  };
  auto fetch = [&](uint32_t dst, const __nv_bfloat16* src, bool live) {
    const uint32_t n = live ? 16u : 0u;                        // the rest of a tile is zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(live ? src : p.cache), "r"(n) : "memory");
  };
  auto request_k = [&](int slot_l) {
    constexpr int CH = DP / 8;
#pragma unroll
    for (int i = 0; i < TOK * CH / 32; ++i) {
      const int idx = i * 32 + lane, r = idx / CH, c = idx % CH;
      const int slot = __shfl_sync(0xffffffff, slot_l, r);
      fetch(kts + at(r, c, Geo::RK), p.cache + static_cast<long long>(slot) * p.row + g * p.dim + c * 8, slot >= 0 && c < kc);
    }
  };
  auto request_v = [&](int slot_l) {
    constexpr int CH = DV / 8;
#pragma unroll
    for (int i = 0; i < TOK * CH / 32; ++i) {
      const int idx = i * 32 + lane, r = idx / CH, c = idx % CH;
      const int slot = __shfl_sync(0xffffffff, slot_l, r);
      fetch(vts + at(r, c, Geo::RV), p.cache + static_cast<long long>(slot) * p.row + p.G * p.dim + g * p.vdim + c * 8,
            slot >= 0 && c < vc);
    }
  };
  auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };
  auto wait_but_one = [] { asm volatile("cp.async.wait_group 1;" ::: "memory"); };

  int slot_l = -1;
  if (warp < ntiles) {
    slot_l = slot_of(warp);
    request_k(slot_l);
  }
  commit();
  if (warp < ntiles) request_v(slot_l);
  commit();

  const bool appends = s1 == seen.count && ntiles > 0;   // the newest position lies in the last tile of this split
  if (ntiles > 0) {
    const int half = p.rot >> 1;
    if (half) {
      for (int i = tid; i < half; i += SDK_WARPS * 32) rotation_at(len - 1, p.turns[i], &s_sin[i], &s_cos[i]);
      __syncthreads();
    }
    // queries (and the new key) rotated and normed, a warp per head; unused rows are zero
    for (int r = warp; r < SDK_ROWS + 1; r += SDK_WARPS) {
      const bool key = r == SDK_ROWS;
      if (key && !appends) break;
      const __nv_bfloat16* src = prow + (key ? p.k_off + g * p.dim : p.q_off + (h0 + r) * p.dim);
      const bool live = key || r < nh;
      float2 v[DP / 64];
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < DP / 64; ++k) {
        const int i = lane + 32 * k;
        v[k] = make_float2(0.f, 0.f);
        if (live && 2 * i < p.dim) v[k] = sa_ld2(src + 2 * i);
        if (i < half) v[k] = sa_rotate(v[k], s_cos[i], s_sin[i]);
        ss = fmaf(v[k].x, v[k].x, fmaf(v[k].y, v[k].y, ss));
      }
      const float f = p.true_dim ? 1.f / sqrtf(sa_warp_sum(ss) / p.true_dim + p.eps) : 1.f;
#pragma unroll
      for (int k = 0; k < DP / 64; ++k) {
        const int i = lane + 32 * k;
        const float2 w = make_float2(v[k].x * f, v[k].y * f);
        if (key) sa_st2(s_key + 2 * i, w);
        else *reinterpret_cast<uint32_t*>(sq + at(r, i >> 2, Geo::RK) + (i & 3) * 4) = pack_bf16x2(w.x, w.y);
      }
    }
  }
  __syncthreads();

  const int r0 = lane >> 2, cq = (lane & 3) * 2;
  float m_run[2] = {-FLT_MAX, -FLT_MAX}, l_run[2] = {0.f, 0.f};
  float o[NO][4];
#pragma unroll
  for (int j = 0; j < NO; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
  const float sl2 = p.scale * SA_LOG2E;
  float pen[2] = {0.f, 0.f}, far[2] = {0.f, 0.f}, bias[2] = {0.f, 0.f};
#pragma unroll
  for (int u = 0; u < HV; ++u) {
    const int h = r0 + 8 * u;
    if (h >= nh) continue;
    if (!SIG && p.r1) { pen[u] = p.r1[h0 + h]; far[u] = p.r2[h0 + h]; }
    if (SIG && p.head_bias) bias[u] = p.head_bias[h0 + h] * SA_LOG2E;
  }

  if (warp < ntiles) {
    uint32_t qa[KS][4];
    const uint32_t sqs = static_cast<uint32_t>(__cvta_generic_to_shared(sq));
#pragma unroll
    for (int ks = 0; ks < KS; ++ks)
      sa_ldsm_x4(qa[ks], sqs + at((lane & 7) + ((lane >> 3) & 1) * 8, ks * 2 + (lane >> 4), Geo::RK));
#pragma unroll 1
    for (int t = warp; t < ntiles; t += SDK_WARPS) {
      const int place0 = s0 + t * TOK;
      const int nt = s1 - place0 < TOK ? s1 - place0 : TOK;
      const bool more = t + SDK_WARPS < ntiles, newest = appends && t == ntiles - 1;
      const int next_slot = more ? slot_of(t + SDK_WARPS) : -1;
      wait_but_one();
      __syncwarp();
      const int new_row = s1 - 1 - place0;
      const int new_slot = newest && hb == 0 ? p.new_slots[b] : -1;
      __nv_bfloat16* store = p.cache + static_cast<long long>(new_slot < 0 ? 0 : new_slot) * p.row;
      if (newest) {
        // the cache row of the newest position is stale: take the key from here, and store it
        for (int c = lane; c < kc; c += 32) {
          const uint4 v = *reinterpret_cast<const uint4*>(s_key + c * 8);
          *reinterpret_cast<uint4*>(kt + at(new_row, c, Geo::RK)) = v;
          if (new_slot >= 0) *reinterpret_cast<uint4*>(store + g * p.dim + c * 8) = v;
        }
        __syncwarp();
      }
      float sc[NT][4];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll
        for (int kp = 0; kp < KS / 2; ++kp) {
          uint32_t kb[4];
          sa_ldsm_x4(kb, kts + at(j * 8 + (lane & 7), kp * 4 + (lane >> 3), Geo::RK));
          sa_mma(sc[j], qa[2 * kp], kb[0], kb[1]);
          sa_mma(sc[j], qa[2 * kp + 1], kb[2], kb[3]);
        }
      }
      __syncwarp();                                  // every lane is done with the keys before they are refilled
      if (more) request_k(next_slot);
      commit();
      if (SIG) {
#pragma unroll
        for (int j = 0; j < NT; ++j) {
#pragma unroll
          for (int e = 0; e < 2 * HV; ++e) {
            const float z = fmaf(sc[j][e], sl2, bias[e >> 1]);
            sc[j][e] = j * 8 + cq + (e & 1) < nt ? __fdividef(1.f, 1.f + ex2(fminf(-z, 120.f))) : 0.f;
          }
        }
      } else {
        float mx[2] = {-FLT_MAX, -FLT_MAX};
#pragma unroll
        for (int j = 0; j < NT; ++j) {
#pragma unroll
          for (int e = 0; e < 2 * HV; ++e) {
            const int ti = j * 8 + cq + (e & 1), u = e >> 1;
            float v = sc[j][e] * sl2;
            if (p.r1) v = fmaf(-pen[u], __log2f(fmaf(far[u], static_cast<float>(len - 1 - seen.position(place0 + ti)), 1.f)), v);
            sc[j][e] = ti < nt ? v : -FLT_MAX;
            mx[u] = fmaxf(mx[u], sc[j][e]);
          }
        }
        float resc[2] = {1.f, 1.f};
#pragma unroll
        for (int u = 0; u < HV; ++u) {
          mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffff, mx[u], 1));
          mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffff, mx[u], 2));
          const float mn = fmaxf(m_run[u], mx[u]);
          resc[u] = ex2(m_run[u] - mn);
          m_run[u] = mn;
          l_run[u] *= resc[u];
        }
        if (ONE8) resc[1] = resc[0];
        if (__any_sync(0xffffffff, resc[0] != 1.f || resc[1] != 1.f)) {
#pragma unroll
          for (int j = 0; j < NO; ++j) { o[j][0] *= resc[0]; o[j][1] *= resc[0]; o[j][2] *= resc[1]; o[j][3] *= resc[1]; }
        }
#pragma unroll
        for (int j = 0; j < NT; ++j) {
#pragma unroll
          for (int e = 0; e < 2 * HV; ++e) {
            sc[j][e] = sc[j][e] == -FLT_MAX ? 0.f : ex2(sc[j][e] - m_run[e >> 1]);
            l_run[e >> 1] += sc[j][e];
          }
        }
      }
      uint32_t ph[NT / 2][4], pl[NT / 2][4];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int a = (j & 1) * 2;
        ph[j >> 1][a] = pack_bf16x2(sc[j][0], sc[j][1]);
        if (ONE8) {
          ph[j >> 1][a + 1] = pack_bf16x2(sa_rest(sc[j][0]), sa_rest(sc[j][1]));
        } else {
          ph[j >> 1][a + 1] = pack_bf16x2(sc[j][2], sc[j][3]);
          pl[j >> 1][a] = pack_bf16x2(sa_rest(sc[j][0]), sa_rest(sc[j][1]));
          pl[j >> 1][a + 1] = pack_bf16x2(sa_rest(sc[j][2]), sa_rest(sc[j][3]));
        }
      }
      wait_but_one();
      __syncwarp();
      if (newest) {
        for (int c = lane; c < vc; c += 32) {
          const uint4 v = *reinterpret_cast<const uint4*>(prow + p.v_off + g * p.vdim + c * 8);
          *reinterpret_cast<uint4*>(vt + at(new_row, c, Geo::RV)) = v;
          if (new_slot >= 0) *reinterpret_cast<uint4*>(store + p.G * p.dim + g * p.vdim + c * 8) = v;
        }
        __syncwarp();
      }
#pragma unroll
      for (int kk = 0; kk < NT / 2; ++kk) {
#pragma unroll
        for (int np = 0; np < NO / 2; ++np) {
          uint32_t vb[4];
          sa_ldsm_x4_t(vb, vts + at(kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, np * 2 + (lane >> 4), Geo::RV));
          sa_mma(o[2 * np], ph[kk], vb[0], vb[1]);
          sa_mma(o[2 * np + 1], ph[kk], vb[2], vb[3]);
          if (!ONE8) {
            sa_mma(o[2 * np], pl[kk], vb[0], vb[1]);
            sa_mma(o[2 * np + 1], pl[kk], vb[2], vb[3]);
          }
        }
      }
      __syncwarp();
      if (more) request_v(next_slot);
      commit();
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  if (!SIG) {
#pragma unroll
    for (int u = 0; u < HV; ++u) {
      l_run[u] += __shfl_xor_sync(0xffffffff, l_run[u], 1);
      l_run[u] += __shfl_xor_sync(0xffffffff, l_run[u], 2);
    }
  }
  __syncthreads();
  float* o_all = reinterpret_cast<float*>(sd_smem);   // [warp][16][DV]
  if (!SIG && (lane & 3) == 0) {
    m_all[warp][r0] = m_run[0]; l_all[warp][r0] = l_run[0];
    if (!ONE8) { m_all[warp][r0 + 8] = m_run[1]; l_all[warp][r0 + 8] = l_run[1]; }
  }
#pragma unroll
  for (int j = 0; j < NO; ++j) {
    float* dst = o_all + (warp * SDK_ROWS + r0) * DV + j * 8 + cq;
    if (ONE8) {
      *reinterpret_cast<float2*>(dst) = make_float2(o[j][0] + o[j][2], o[j][1] + o[j][3]);
    } else {
      *reinterpret_cast<float2*>(dst) = make_float2(o[j][0], o[j][1]);
      *reinterpret_cast<float2*>(dst + 8 * DV) = make_float2(o[j][2], o[j][3]);
    }
  }
  __syncthreads();
  for (int i = tid; i < nh * p.vdim; i += SDK_WARPS * 32) {
    const int r = i / p.vdim, d = i - r * p.vdim;
    float mm = 0.f, acc = 0.f, ls = 0.f;
    if (SIG) {
#pragma unroll
      for (int w = 0; w < SDK_WARPS; ++w) acc += o_all[(w * SDK_ROWS + r) * DV + d];
    } else {
      mm = -FLT_MAX;
#pragma unroll
      for (int w = 0; w < SDK_WARPS; ++w) mm = fmaxf(mm, m_all[w][r]);
#pragma unroll
      for (int w = 0; w < SDK_WARPS; ++w) {
        const float f = m_all[w][r] == -FLT_MAX ? 0.f : ex2(m_all[w][r] - mm);
        acc += o_all[(w * SDK_ROWS + r) * DV + d] * f;
        ls += l_all[w][r] * f;
      }
    }
    if (p.nsplit == 1) {
      const float f = SIG ? p.out_scale : ls > 0.f ? p.out_scale / ls : 0.f;
      p.out[b * p.o_ld + static_cast<long long>(h0 + r) * p.vdim + d] = __float2bfloat16(acc * f);
    } else {
      float* dst = p.scratch + ((static_cast<long long>(b) * p.H + h0 + r) * p.nsplit + split) * (p.vdim + 2);
      dst[d] = acc;
      if (!SIG && d == 0) { dst[p.vdim] = mm; dst[p.vdim + 1] = ls; }
    }
  }
}

constexpr int SM_THREADS = 128;
// grid (request, head).  Scratch rows are [values | running max | running sum], in the log2 domain; SIG: the values alone.
template <bool SIG>
__global__ void __launch_bounds__(SM_THREADS) scored_merge_kernel(const ScoredDecodeParams p) {
  __shared__ float s_w[SDK_MAX_SPLITS];
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, V = p.vdim;
  const float* base = p.scratch + (static_cast<long long>(b) * p.H + h) * p.nsplit * (V + 2);
  const SeenKeys seen(p.ctx_len[b], p.window, p.keep);
  int ns = (seen.count + p.split_tokens - 1) / p.split_tokens;
  ns = ns < 1 ? 1 : (ns > p.nsplit ? p.nsplit : ns);
  if (SIG) {
    for (int s = tid; s < ns; s += SM_THREADS) s_w[s] = p.out_scale;
  } else if (tid < 32) {
    const float* src = base + V;
    float mm = -FLT_MAX, l = 0.f;
    for (int s = tid; s < ns; s += 32) mm = fmaxf(mm, src[static_cast<long long>(s) * (V + 2)]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mm = fmaxf(mm, __shfl_xor_sync(0xffffffff, mm, o));
    for (int s = tid; s < ns; s += 32) {
      const float ms = src[static_cast<long long>(s) * (V + 2)];
      const float w = ms == -FLT_MAX ? 0.f : ex2(ms - mm);
      s_w[s] = w;
      l += src[static_cast<long long>(s) * (V + 2) + 1] * w;
    }
    l = sa_warp_sum(l);
    const float f = l > 0.f ? p.out_scale / l : 0.f;
    for (int s = tid; s < ns; s += 32) s_w[s] *= f;
  }
  __syncthreads();
  for (int d = tid; d < V; d += SM_THREADS) {
    float v = 0.f;
#pragma unroll 4
    for (int s = 0; s < ns; ++s) v = fmaf(base[static_cast<long long>(s) * (V + 2) + d], s_w[s], v);
    p.out[b * p.o_ld + static_cast<long long>(h) * V + d] = __float2bfloat16(v);
  }
}

// About one wave of CTAs, never finer than SDK_MIN_SPLIT tokens.  Depends on host values only.
inline void scored_splits(int B, int H, int G, int span, int* nsplit, int* split_tokens) {
  const int groups = B * G * ((H / G + SDK_ROWS - 1) / SDK_ROWS);
  int ns = (span + SDK_MIN_SPLIT - 1) / SDK_MIN_SPLIT;
  int want = scored_decode_target_ctas() / (groups > 0 ? groups : 1);
  if (want < 1) want = 1;
  if (want > SDK_MAX_SPLITS) want = SDK_MAX_SPLITS;
  if (ns < 1) ns = 1;
  if (want < ns) ns = want;
  int st = ((span + ns - 1) / ns + 31) / 32 * 32;
  if (st < SDK_MIN_SPLIT) st = SDK_MIN_SPLIT;
  ns = (span + st - 1) / st;
  *nsplit = ns < 1 ? 1 : ns;
  *split_tokens = st;
}

inline int scored_span(int window, int keep, int max_ctx) {
  const long long s = static_cast<long long>(window) + keep;
  return window > 0 && s < max_ctx ? static_cast<int>(s) : max_ctx;
}

template <int DP, int DV, int TOK, bool ONE8, bool SIG>
int launch_sd(const ScoredDecodeParams& p, int B, cudaStream_t st) {
  using Geo = SdGeo<DP, DV, TOK>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(scored_decode_kernel<DP, DV, TOK, ONE8, SIG>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, Geo::SMEM);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured = true;
  }
  const int yb = p.G * ((p.H / p.G + SDK_ROWS - 1) / SDK_ROWS);
  launch_k(scored_decode_kernel<DP, DV, TOK, ONE8, SIG>, dim3(B, yb, p.nsplit), dim3(SDK_WARPS * 32), Geo::SMEM, st, p);
  if (p.nsplit > 1) launch_k(scored_merge_kernel<SIG>, dim3(B, p.H), dim3(SM_THREADS), 0, st, p);
  return launch_status();
}

template <int DP, int DV, int TOK>
int launch_sd_kind(const ScoredDecodeParams& p, int B, bool sig, cudaStream_t st) {
  const bool one8 = p.H / p.G <= 8;
  if (sig) return one8 ? launch_sd<DP, DV, TOK, true, true>(p, B, st) : launch_sd<DP, DV, TOK, false, true>(p, B, st);
  return one8 ? launch_sd<DP, DV, TOK, true, false>(p, B, st) : launch_sd<DP, DV, TOK, false, false>(p, B, st);
}

}  // namespace gk

using namespace gk;

// ptrs: {proj, turns, pos, slots, cache};  turns: with rot;  cache null: keys in place, slots may be null too
// dims: {rows, q_off, k_off, v_off, NQ, NK, D, VC, rot, true_D}
// Offsets, D and VC are multiples of 8, rot is even; cached rows are NK * D + VC elements.  true_D 0: no norm.
GK_EXPORT int gk_head_prep(int is_fp32, void* const* ptrs, long long ld, const int* dims, float eps, void* stream) {
  if (dims[0] == 0) return 0;
  for (int i = 0; i < 10; ++i)
    if (dims[i] < 0 || ((i == 1 || i == 2 || i == 3 || i == 6 || i == 7) && dims[i] % 8)) return -1;
  if (ld % 8 || dims[8] % 2 || dims[8] > dims[6] || dims[8] > SA_MAX_ROT || dims[9] > dims[6] || dims[6] < 8) return -1;
  if ((dims[8] && (!ptrs[1] || !ptrs[2])) || (ptrs[4] && !ptrs[3])) return -1;
  if ((reinterpret_cast<uintptr_t>(ptrs[0]) | reinterpret_cast<uintptr_t>(ptrs[4])) & 15) return -1;
  auto fill = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    HeadPrepParams<T> p;
    p.proj = static_cast<T*>(ptrs[0]); p.ld = ld;
    p.turns = static_cast<const float2*>(ptrs[1]);
    p.pos = static_cast<const int*>(ptrs[2]); p.slots = static_cast<const int*>(ptrs[3]);
    p.cache = static_cast<T*>(ptrs[4]);
    p.q_off = dims[1]; p.k_off = dims[2]; p.v_off = dims[3]; p.NQ = dims[4]; p.NK = dims[5]; p.D = dims[6]; p.VC = dims[7];
    p.rot = dims[8]; p.true_D = dims[9]; p.eps = eps;
    return launch_head_prep(p, dims[0], reinterpret_cast<cudaStream_t>(stream));
  };
  return is_fp32 ? fill(static_cast<float*>(nullptr)) : fill(static_cast<__nv_bfloat16*>(nullptr));
}

// Columns off .. off + n (multiples of 8) of `rows` rows become their silu.
GK_EXPORT int gk_silu_columns(int is_fp32, void* proj, long long ld, int off, int n, int rows, void* stream) {
  if (rows == 0 || n == 0) return 0;
  if (rows < 0 || n < 0 || n % 8 || off < 0 || off % 8 || ld % 8 || (reinterpret_cast<uintptr_t>(proj) & 15)) return -1;
  const int x = (n / 8 + 255) / 256;
  int y = sm_count() * 16 / x;
  y = y < 1 ? 1 : y > rows ? rows : y;
  const dim3 grid(x, y), block(256);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (is_fp32) launch_k(silu_columns_kernel<float>, grid, block, 0, st, static_cast<float*>(proj), ld, off, n, rows);
  else launch_k(silu_columns_kernel<__nv_bfloat16>, grid, block, 0, st, static_cast<__nv_bfloat16*>(proj), ld, off, n, rows);
  return launch_status();
}

GK_EXPORT void gk_scored_set_target_ctas(int n) { scored_decode_target_ctas() = n > 0 ? n : 444; }

// 1 when a kernel is built for keys of `dim` and values of `vdim` columns
GK_EXPORT int gk_scored_decode_supported(int dim, int vdim) { return dim >= 1 && dim <= 128 && vdim >= 1 && vdim <= 256; }

GK_EXPORT long long gk_scored_decode_scratch(int B, int H, int G, int vdim, int window, int keep, int max_ctx) {
  int ns, st;
  scored_splits(B, H, G, scored_span(window, keep, max_ctx), &ns, &st);
  return ns > 1 ? static_cast<long long>(B) * H * ns * (vdim + 2) : 0;
}

// One new token per request; max_ctx bounds every ctx_len[b].  sigmoid: sigmoids in place of the softmax.
// ptrs: {proj, cache, tables, ctx_len, new_slots, turns, r1, r2, head_bias, out, scratch};  lds: {ld, o_ld}
// dims: {B, H, G, dim, vdim, rot, true_dim, q_off, k_off, v_off, row, block_size, max_blocks, max_ctx, window, keep, sigmoid}
// floats: {scale, out_scale, eps};  true_dim 0: queries and keys are not normed;  window 0: unlimited
GK_EXPORT int gk_scored_decode(void* const* ptrs, const long long* lds, const int* dims, const float* floats, void* stream) {
  const int B = dims[0], H = dims[1], G = dims[2], dim = dims[3], vdim = dims[4];
  if (!gk_scored_decode_supported(dim, vdim) || G < 1 || H % G || dim % 8 || vdim % 8 || dims[5] % 2 || dims[5] > dim) return -1;
  if (dims[6] < 0 || dims[6] > dim || dims[14] < 0 || dims[15] < 0 || dims[11] < 1 || (dims[5] && !ptrs[5])) return -1;
  if (lds[0] % 8 || dims[7] % 8 || dims[8] % 8 || dims[9] % 8 || dims[10] % 8 || dims[10] < G * (dim + vdim)) return -1;
  if ((ptrs[6] != nullptr) != (ptrs[7] != nullptr) || (dims[16] ? ptrs[6] != nullptr : ptrs[8] != nullptr)) return -1;
  if ((reinterpret_cast<uintptr_t>(ptrs[0]) | reinterpret_cast<uintptr_t>(ptrs[1])) & 15) return -1;
  if (B == 0) return 0;
  ScoredDecodeParams p;
  p.proj = static_cast<const __nv_bfloat16*>(ptrs[0]); p.ld = lds[0];
  p.cache = static_cast<__nv_bfloat16*>(ptrs[1]);
  p.tables = static_cast<const int*>(ptrs[2]); p.ctx_len = static_cast<const int*>(ptrs[3]);
  p.new_slots = static_cast<const int*>(ptrs[4]);
  p.turns = static_cast<const float2*>(ptrs[5]);
  p.r1 = static_cast<const float*>(ptrs[6]); p.r2 = static_cast<const float*>(ptrs[7]);
  p.head_bias = static_cast<const float*>(ptrs[8]);
  p.out = static_cast<__nv_bfloat16*>(ptrs[9]); p.o_ld = lds[1];
  p.scratch = static_cast<float*>(ptrs[10]);
  p.H = H; p.G = G; p.dim = dim; p.vdim = vdim; p.rot = dims[5]; p.true_dim = dims[6];
  p.q_off = dims[7]; p.k_off = dims[8]; p.v_off = dims[9]; p.row = dims[10];
  p.block_size = dims[11]; p.max_blocks = dims[12]; p.window = dims[14]; p.keep = dims[15];
  p.scale = floats[0]; p.out_scale = floats[1]; p.eps = floats[2];
  scored_splits(B, H, G, scored_span(p.window, p.keep, dims[13]), &p.nsplit, &p.split_tokens);
  if (p.nsplit > 1 && !p.scratch) return -2;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const bool sig = dims[16] != 0;
  if (dim <= 64) {
    if (vdim <= 64) return launch_sd_kind<64, 64, 32>(p, B, sig, st);
    if (vdim <= 128) return launch_sd_kind<64, 128, 32>(p, B, sig, st);
    return launch_sd_kind<64, 256, 16>(p, B, sig, st);
  }
  if (vdim <= 64) return launch_sd_kind<128, 64, 32>(p, B, sig, st);
  if (vdim <= 128) return launch_sd_kind<128, 128, 32>(p, B, sig, st);
  return launch_sd_kind<128, 256, 16>(p, B, sig, st);
}
