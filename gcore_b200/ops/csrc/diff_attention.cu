// Differential attention of served decoders around the prompt kernel (diff_prefill.cu): heads subtract two softmax maps over
// the same values, o = a1 - lambda * a2, normed over the head, scaled, gated.  A cached row is [2G keys | G values]; head h's
// maps read keys 2g and 2g + 1 and value g = h / (H / G).
//   * rotate_append_kernel   a packed projection row: queries rotated in place, rotated keys and the values to their slot;
//   * diff_decode_kernel     one new token per request, bf16, KV splits, on mma.sync tiles (a group of heads is far below the
//                            64-row minimum of a tcgen05 instruction).  Rows 0-7 of a tile are the first maps of up to eight
//                            heads, rows 8-15 their second maps.  The score contraction runs over both keys at once with
//                            queries that are zero in the other map's half, so one 16-row probability tile multiplies the
//                            values once for both maps.  Rotation and append of the new token are part of it.
//   * diff_merge_kernel      merges the KV splits of both maps and finishes the head;
//   * diff_finish_kernel     finishes heads whose maps (or difference) lie in 32-bit rows.
// Probabilities stay 32-bit: for the tensor core they are split into two bf16 terms (rounded value, remainder).
#include "ptx.cuh"
#include "host_utils.h"
#include "rotary.cuh"
#include "row_ops.cuh"
#include <cuda_bf16.h>
#include <float.h>
#include <type_traits>

namespace gk {

constexpr int DA_MAX_ROT = 256;

__device__ __forceinline__ float2 da_ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 da_ld2(const __nv_bfloat16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
__device__ __forceinline__ void da_st2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void da_st2(__nv_bfloat16* p, float2 v) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y);
}
__device__ __forceinline__ float da_f(float v) { return v; }
__device__ __forceinline__ float da_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void da_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void da_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float2 da_rotate(float2 v, float c, float s) { return make_float2(v.x * c - v.y * s, v.y * c + v.x * s); }

template <typename T>
struct RotateAppendParams {
  T* proj;                 // packed projection rows
  long long ld;
  int q_off, k_off, v_off; // NQ queries, NK keys of D columns each, VC value columns
  int NQ, NK, D, VC, rot;
  const float2* turns;     // [rot / 2] turns per position: value, remainder
  const int *pos, *slots;  // cache slot of every row; negative: not stored
  T* cache;                // rows of NK * D + VC
  float magnitude;
};

// One CTA per row.
template <typename T>
__global__ void __launch_bounds__(128) rotate_append_kernel(const RotateAppendParams<T> p) {
  __shared__ float s_cos[DA_MAX_ROT / 2], s_sin[DA_MAX_ROT / 2];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, tid = threadIdx.x, half = p.rot >> 1;
  T* pr = p.proj + row * p.ld;
  const int pos = p.pos[row], slot = p.slots[row];
  for (int i = tid; i < half; i += 128) {
    float s, c;
    rotation_at(pos, p.turns[i], &s, &c);
    s_cos[i] = c * p.magnitude;
    s_sin[i] = s * p.magnitude;
  }
  __syncthreads();
  for (int i = tid; i < p.NQ * half; i += 128) {
    const int h = i / half, j = i - h * half;
    T* q = pr + p.q_off + static_cast<long long>(h) * p.D + 2 * j;
    da_st2(q, da_rotate(da_ld2(q), s_cos[j], s_sin[j]));
  }
  if (slot < 0) return;
  const int hd = p.D >> 1, keys = p.NK * hd, all = keys + (p.VC >> 1);
  T* dst = p.cache + static_cast<long long>(slot) * (p.NK * p.D + p.VC);
  for (int i = tid; i < all; i += 128) {
    float2 v;
    if (i < keys) {
      const int j = i % hd;
      v = da_ld2(pr + p.k_off + 2 * i);
      if (j < half) v = da_rotate(v, s_cos[j], s_sin[j]);
    } else {
      v = da_ld2(pr + p.v_off + 2 * (i - keys));
    }
    da_st2(dst + 2 * i, v);
  }
}

// ---------------------------------------------------------------------------------------------------- finishing a head
// Warp per (row, head).  MAPS 2: a holds both maps [row, H, 2, V]; 1: their difference [row, H, V].
template <typename T, int MAPS>
__global__ void __launch_bounds__(128) diff_finish_kernel(const float* __restrict__ a, const T* __restrict__ gate,
                                                          long long gate_ld, T* __restrict__ out, long long o_ld,
                                                          const float* __restrict__ lam, int rows, int H, int V, int true_v,
                                                          float out_scale, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  const long long item = static_cast<long long>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  if (item >= static_cast<long long>(rows) * H) return;
  const long long row = item / H;
  const int h = static_cast<int>(item - row * H), lane = threadIdx.x & 31;
  const float* src = a + item * MAPS * V;
  const float lm = MAPS == 2 ? *lam : 0.f;
  float ss = 0.f;
  for (int d = lane; d < V; d += 32) {
    const float v = MAPS == 2 ? src[d] - lm * src[V + d] : src[d];
    ss = fmaf(v, v, ss);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffff, ss, o);
  const float f = out_scale / (sqrtf(ss / true_v + eps) * (1.f + expf(-da_f(gate[row * gate_ld + h]))));
  T* dst = out + row * o_ld + static_cast<long long>(h) * V;
  for (int d = lane; d < V; d += 32) da_st(dst + d, (MAPS == 2 ? src[d] - lm * src[V + d] : src[d]) * f);
}

// ---------------------------------------------------------------------------------------------------- bf16 decode
__device__ __forceinline__ void da_ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void da_ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void da_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                       uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float da_rest(float v) { return v - __bfloat162float(__float2bfloat16(v)); }

constexpr int DD_WARPS = 4;
constexpr int DD_HEADS = 8;        // heads per CTA; the tiles' 16 rows are their two maps
constexpr int DD_MIN_SPLIT = 128;
constexpr int DD_MAX_SPLITS = 256;
inline int& diff_decode_target_ctas() {
  static int n = 444;
  return n;
}

struct DiffDecodeParams {
  const __nv_bfloat16* proj;   // packed rows, one per request, not rotated yet
  long long ld;
  int q_off, k_off, v_off, gate_off;
  __nv_bfloat16* cache;        // rows of `row` elements: 2G keys of `dim`, G values of `vdim` columns
  int row;
  const int* tables;
  int max_blocks, block_size;
  const int* ctx_len;          // counts the new token; 0: inactive
  const int* new_slots;
  const float2* turns;
  const float* lam;
  __nv_bfloat16* out;
  long long o_ld;
  float* scratch;              // [B, H, 2, nsplit, vdim + 2]
  int H, G, dim, vdim, true_vdim, rot, nsplit, split_tokens;
  float scale, magnitude, out_scale, eps;
};

// DP: columns of a key tile per map (dim <= DP), DV: of a value tile, TOK: tokens per warp tile.
template <int DP, int DV, int TOK>
struct DdGeo {
  static constexpr int RK = 4 * DP, RV = 2 * DV;                     // bytes of a key / value tile row
  static constexpr int WARP = TOK * (RK + RV);
  static constexpr int TILES = DD_WARPS * WARP, MERGE = DD_WARPS * 16 * DV * 4;
  static constexpr int SMEM = TILES > MERGE ? TILES : MERGE;
  static constexpr int CTAS = SMEM <= 56 * 1024 && DV <= 128 ? 4 : SMEM <= 72 * 1024 && DV <= 128 ? 3 : 2;
};

// grid (request, kv head x blocks of 8 heads, split)
template <int DP, int DV, int TOK>
__global__ void __launch_bounds__(DD_WARPS * 32, (DdGeo<DP, DV, TOK>::CTAS)) diff_decode_kernel(const DiffDecodeParams p) {
  using Geo = DdGeo<DP, DV, TOK>;
  constexpr int NT = TOK / 8;          // score tiles of 8 tokens
  constexpr int NO = DV / 8;           // output tiles of 8 columns
  constexpr int KS = DP / 16;          // k-steps of one map
  extern __shared__ __align__(128) uint8_t dd_smem[];
  __shared__ float m_all[DD_WARPS][16], l_all[DD_WARPS][16];
  __shared__ float s_cos[DP / 2], s_sin[DP / 2];

  pdl_launch_dependents();
  pdl_wait();
  const int grp = p.H / p.G, hblocks = (grp + DD_HEADS - 1) / DD_HEADS;
  const int b = blockIdx.x, g = blockIdx.y / hblocks, hb = blockIdx.y % hblocks, split = blockIdx.z;
  const int h0 = g * grp + hb * DD_HEADS;
  const int nh = grp - hb * DD_HEADS < DD_HEADS ? grp - hb * DD_HEADS : DD_HEADS;
  const int len = p.ctx_len[b];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int s0 = split * p.split_tokens;
  if (split > 0 && s0 >= len) return;                          // dead split: the merge kernel skips it
  const int s1 = s0 + p.split_tokens < len ? s0 + p.split_tokens : len;
  const int ntiles = s1 > s0 ? (s1 - s0 + TOK - 1) / TOK : 0;
  const __nv_bfloat16* prow = p.proj + b * p.ld;
  const int kc = p.dim >> 3, vc = p.vdim >> 3;                 // 16-byte chunks in use

  uint8_t* kt = dd_smem + warp * Geo::WARP;
  uint8_t* vt = kt + TOK * Geo::RK;
  const uint32_t kts = static_cast<uint32_t>(__cvta_generic_to_shared(kt));
  const uint32_t vts = static_cast<uint32_t>(__cvta_generic_to_shared(vt));
  // chunk ch of row r: the low three chunk bits are xor-ed with the row, so an ldmatrix is free of bank conflicts
  auto at = [](int r, int ch, int row_bytes) { return r * row_bytes + (((ch & ~7) | ((ch ^ r) & 7)) << 4); };
  auto slot_of = [&](int t) -> int {
    const int tok = s0 + t * TOK + (lane < TOK ? lane : TOK - 1);
    return tok < s1 ? p.tables[static_cast<long long>(b) * p.max_blocks + tok / p.block_size] * p.block_size +
                          tok % p.block_size
                    : -1;
  };
  auto fetch = [&](uint32_t dst, const __nv_bfloat16* src, bool live) {
    const uint32_t n = live ? 16u : 0u;                        // the rest of a tile is zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(live ? src : p.cache), "r"(n) : "memory");
  };
  auto request_k = [&](int slot_l) {
    constexpr int CH = DP / 4;                                 // chunks of a row, both maps
#pragma unroll
    for (int i = 0; i < TOK * CH / 32; ++i) {
      const int idx = i * 32 + lane, r = idx / CH, ch = idx % CH, m = ch / (DP / 8), c = ch % (DP / 8);
      const int slot = __shfl_sync(0xffffffff, slot_l, r);
      fetch(kts + at(r, ch, Geo::RK), p.cache + static_cast<long long>(slot) * p.row + (2 * g + m) * p.dim + c * 8,
            slot >= 0 && c < kc);
    }
  };
  auto request_v = [&](int slot_l) {
    constexpr int CH = DV / 8;
#pragma unroll
    for (int i = 0; i < TOK * CH / 32; ++i) {
      const int idx = i * 32 + lane, r = idx / CH, c = idx % CH;
      const int slot = __shfl_sync(0xffffffff, slot_l, r);
      fetch(vts + at(r, c, Geo::RV),
            p.cache + static_cast<long long>(slot) * p.row + 2 * p.G * p.dim + g * p.vdim + c * 8, slot >= 0 && c < vc);
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

  const int half = p.rot >> 1;
  for (int i = tid; i < half; i += DD_WARPS * 32) {
    float s, c;
    rotation_at(len - 1, p.turns[i], &s, &c);
    s_cos[i] = c * p.magnitude;
    s_sin[i] = s * p.magnitude;
  }
  __syncthreads();
  auto rotated = [&](uint32_t v, int pair) -> uint32_t {
    if (pair >= half) return v;
    const float2 r = da_rotate(__bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&v)), s_cos[pair], s_sin[pair]);
    return pack_bf16x2(r.x, r.y);
  };

  const int r0 = lane >> 2, cq = (lane & 3) * 2;
  float m_run[2] = {-FLT_MAX, -FLT_MAX}, l_run[2] = {0.f, 0.f};
  float o[NO][4];
#pragma unroll
  for (int j = 0; j < NO; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
  const float sl2 = p.scale * 1.4426950408889634f;
  const bool appends = s1 == len && ntiles > 0;   // the newest position lies in the last tile of this split

  if (warp < ntiles) {
    // the queries as A fragments: head r0's map m fills row r0 + 8 m only
    uint32_t qa[2][KS][2];
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const __nv_bfloat16* q = prow + p.q_off + static_cast<long long>(2 * (h0 + r0) + m) * p.dim;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int col = ks * 16 + e * 8 + cq;
          qa[m][ks][e] = r0 < nh && col < p.dim ? rotated(*reinterpret_cast<const uint32_t*>(q + col), col >> 1) : 0u;
        }
      }
    }
#pragma unroll 1
    for (int t = warp; t < ntiles; t += DD_WARPS) {
      const int tok0 = s0 + t * TOK;
      const int nt = s1 - tok0 < TOK ? s1 - tok0 : TOK;
      const bool more = t + DD_WARPS < ntiles, newest = appends && t == ntiles - 1;
      const int next_slot = more ? slot_of(t + DD_WARPS) : -1;
      wait_but_one();
      __syncwarp();
      const int new_row = len - 1 - tok0;
      const int new_slot = newest && hb == 0 ? p.new_slots[b] : -1;
      __nv_bfloat16* store = p.cache + static_cast<long long>(new_slot < 0 ? 0 : new_slot) * p.row;
      if (newest) {
        // the cache row of the newest position is stale: take the keys from the projection, and store them
        for (int i = lane; i < 2 * kc; i += 32) {
          const int m = i / kc, c = i - m * kc;
          uint4 v = *reinterpret_cast<const uint4*>(prow + p.k_off + (2 * g + m) * p.dim + c * 8);
          v.x = rotated(v.x, 4 * c); v.y = rotated(v.y, 4 * c + 1);
          v.z = rotated(v.z, 4 * c + 2); v.w = rotated(v.w, 4 * c + 3);
          *reinterpret_cast<uint4*>(kt + at(new_row, m * (DP / 8) + c, Geo::RK)) = v;
          if (new_slot >= 0) *reinterpret_cast<uint4*>(store + (2 * g + m) * p.dim + c * 8) = v;
        }
        __syncwarp();
      }
      float sc[NT][4];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll
        for (int kp = 0; kp < KS; ++kp) {            // pairs of k-steps over both maps
          uint32_t kb[4];
          da_ldsm_x4(kb, kts + at(j * 8 + (lane & 7), kp * 4 + (lane >> 3), Geo::RK));
          const int m = kp / (KS / 2), ks = 2 * (kp % (KS / 2));
          if (m == 0) {
            da_mma(sc[j], qa[0][ks][0], 0u, qa[0][ks][1], 0u, kb[0], kb[1]);
            da_mma(sc[j], qa[0][ks + 1][0], 0u, qa[0][ks + 1][1], 0u, kb[2], kb[3]);
          } else {
            da_mma(sc[j], 0u, qa[1][ks][0], 0u, qa[1][ks][1], kb[0], kb[1]);
            da_mma(sc[j], 0u, qa[1][ks + 1][0], 0u, qa[1][ks + 1][1], kb[2], kb[3]);
          }
        }
      }
      __syncwarp();                                  // every lane is done with the keys before they are refilled
      if (more) request_k(next_slot);
      commit();
      float mx[2] = {-FLT_MAX, -FLT_MAX};
#pragma unroll
      for (int j = 0; j < NT; ++j) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float v = j * 8 + cq + (e & 1) < nt ? sc[j][e] * sl2 : -FLT_MAX;
          sc[j][e] = v;
          mx[e >> 1] = fmaxf(mx[e >> 1], v);
        }
      }
      float resc[2];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffff, mx[u], 1));
        mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffff, mx[u], 2));
        const float mn = fmaxf(m_run[u], mx[u]);
        resc[u] = ex2(m_run[u] - mn);
        m_run[u] = mn;
        l_run[u] *= resc[u];
      }
      if (__any_sync(0xffffffff, resc[0] != 1.f || resc[1] != 1.f)) {
#pragma unroll
        for (int j = 0; j < NO; ++j) { o[j][0] *= resc[0]; o[j][1] *= resc[0]; o[j][2] *= resc[1]; o[j][3] *= resc[1]; }
      }
      uint32_t ph[NT / 2][4], pl[NT / 2][4];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        float pv[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          pv[e] = sc[j][e] == -FLT_MAX ? 0.f : ex2(sc[j][e] - m_run[e >> 1]);
          l_run[e >> 1] += pv[e];
        }
        ph[j >> 1][(j & 1) * 2] = pack_bf16x2(pv[0], pv[1]);
        ph[j >> 1][(j & 1) * 2 + 1] = pack_bf16x2(pv[2], pv[3]);
        pl[j >> 1][(j & 1) * 2] = pack_bf16x2(da_rest(pv[0]), da_rest(pv[1]));
        pl[j >> 1][(j & 1) * 2 + 1] = pack_bf16x2(da_rest(pv[2]), da_rest(pv[3]));
      }
      wait_but_one();
      __syncwarp();
      if (newest) {
        for (int c = lane; c < vc; c += 32) {
          const uint4 v = *reinterpret_cast<const uint4*>(prow + p.v_off + g * p.vdim + c * 8);
          *reinterpret_cast<uint4*>(vt + at(new_row, c, Geo::RV)) = v;
          if (new_slot >= 0) *reinterpret_cast<uint4*>(store + 2 * p.G * p.dim + g * p.vdim + c * 8) = v;
        }
        __syncwarp();
      }
#pragma unroll
      for (int kk = 0; kk < NT / 2; ++kk) {
#pragma unroll
        for (int np = 0; np < NO / 2; ++np) {
          uint32_t vb[4];
          da_ldsm_x4_t(vb, vts + at(kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, np * 2 + (lane >> 4), Geo::RV));
          da_mma(o[2 * np], ph[kk][0], ph[kk][1], ph[kk][2], ph[kk][3], vb[0], vb[1]);
          da_mma(o[2 * np + 1], ph[kk][0], ph[kk][1], ph[kk][2], ph[kk][3], vb[2], vb[3]);
          da_mma(o[2 * np], pl[kk][0], pl[kk][1], pl[kk][2], pl[kk][3], vb[0], vb[1]);
          da_mma(o[2 * np + 1], pl[kk][0], pl[kk][1], pl[kk][2], pl[kk][3], vb[2], vb[3]);
        }
      }
      __syncwarp();
      if (more) request_v(next_slot);
      commit();
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    l_run[u] += __shfl_xor_sync(0xffffffff, l_run[u], 1);
    l_run[u] += __shfl_xor_sync(0xffffffff, l_run[u], 2);
  }
  __syncthreads();
  float* o_all = reinterpret_cast<float*>(dd_smem);   // [warp][16][DV]
  if ((lane & 3) == 0) {
    m_all[warp][r0] = m_run[0]; l_all[warp][r0] = l_run[0];
    m_all[warp][r0 + 8] = m_run[1]; l_all[warp][r0 + 8] = l_run[1];
  }
#pragma unroll
  for (int j = 0; j < NO; ++j) {
    *reinterpret_cast<float2*>(o_all + (warp * 16 + r0) * DV + j * 8 + cq) = make_float2(o[j][0], o[j][1]);
    *reinterpret_cast<float2*>(o_all + (warp * 16 + r0 + 8) * DV + j * 8 + cq) = make_float2(o[j][2], o[j][3]);
  }
  __syncthreads();
  for (int i = tid; i < 16 * p.vdim; i += DD_WARPS * 32) {
    const int r = i / p.vdim, d = i - r * p.vdim;
    if ((r & 7) >= nh) continue;
    float mm = -FLT_MAX;
#pragma unroll
    for (int w = 0; w < DD_WARPS; ++w) mm = fmaxf(mm, m_all[w][r]);
    float acc = 0.f, ls = 0.f;
#pragma unroll
    for (int w = 0; w < DD_WARPS; ++w) {
      const float f = m_all[w][r] == -FLT_MAX ? 0.f : ex2(m_all[w][r] - mm);
      acc += o_all[(w * 16 + r) * DV + d] * f;
      ls += l_all[w][r] * f;
    }
    if (p.nsplit == 1) {
      o_all[r * DV + d] = ls > 0.f ? acc / ls : 0.f;   // read by this thread only
    } else {
      const long long map = (static_cast<long long>(b) * p.H + h0 + (r & 7)) * 2 + (r >> 3);
      float* dst = p.scratch + (map * p.nsplit + split) * (p.vdim + 2);
      dst[d] = acc;
      if (d == 0) { dst[p.vdim] = mm; dst[p.vdim + 1] = ls; }
    }
  }
  if (p.nsplit > 1) return;
  __syncthreads();
  const float lam = *p.lam;
  for (int r = warp; r < nh; r += DD_WARPS) {
    const float *a1 = o_all + r * DV, *a2 = o_all + (r + 8) * DV;
    float ss = 0.f;
    for (int d = lane; d < p.vdim; d += 32) {
      const float v = a1[d] - lam * a2[d];
      ss = fmaf(v, v, ss);
    }
#pragma unroll
    for (int s = 16; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffff, ss, s);
    const float z = __bfloat162float(prow[p.gate_off + h0 + r]);
    const float f = p.out_scale / (sqrtf(ss / p.true_vdim + p.eps) * (1.f + expf(-z)));
    __nv_bfloat16* dst = p.out + b * p.o_ld + static_cast<long long>(h0 + r) * p.vdim;
    for (int d = lane; d < p.vdim; d += 32) dst[d] = __float2bfloat16((a1[d] - lam * a2[d]) * f);
  }
}

constexpr int DM_THREADS = 128;
// grid (request, head).  Scratch rows are [values | running max | running sum], in the log2 domain.
__global__ void __launch_bounds__(DM_THREADS) diff_merge_kernel(const DiffDecodeParams p) {
  __shared__ float s_w[2][DD_MAX_SPLITS];
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, V = p.vdim;
  const float* base = p.scratch + (static_cast<long long>(b) * p.H + h) * 2 * p.nsplit * (V + 2);
  int ns = (p.ctx_len[b] + p.split_tokens - 1) / p.split_tokens;
  ns = ns < 1 ? 1 : (ns > p.nsplit ? p.nsplit : ns);
  if (tid < 64) {                        // a warp per map: the splits' weights
    const int m = tid >> 5;
    const float* src = base + static_cast<long long>(m) * p.nsplit * (V + 2) + V;
    float mm = -FLT_MAX, l = 0.f;
    for (int s = lane; s < ns; s += 32) mm = fmaxf(mm, src[static_cast<long long>(s) * (V + 2)]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mm = fmaxf(mm, __shfl_xor_sync(0xffffffff, mm, o));
    for (int s = lane; s < ns; s += 32) {
      const float ms = src[static_cast<long long>(s) * (V + 2)];
      const float w = ms == -FLT_MAX ? 0.f : ex2(ms - mm);
      s_w[m][s] = w;
      l += src[static_cast<long long>(s) * (V + 2) + 1] * w;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffff, l, o);
    const float f = l > 0.f ? (m == 0 ? 1.f : -*p.lam) / l : 0.f;
    for (int s = lane; s < ns; s += 32) s_w[m][s] *= f;
  }
  __syncthreads();
  float v[2] = {0.f, 0.f}, ss = 0.f;
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int d = tid + k * DM_THREADS;
    if (d < V) {
      const float *p1 = base + d, *p2 = base + static_cast<long long>(p.nsplit) * (V + 2) + d;
#pragma unroll 4
      for (int s = 0; s < ns; ++s) {
        v[k] = fmaf(p1[static_cast<long long>(s) * (V + 2)], s_w[0][s], v[k]);
        v[k] = fmaf(p2[static_cast<long long>(s) * (V + 2)], s_w[1][s], v[k]);
      }
      ss = fmaf(v[k], v[k], ss);
    }
  }
  ss = block_sum2(ss, 0.f, red).x;
  const float z = __bfloat162float(p.proj[b * p.ld + p.gate_off + h]);
  const float f = p.out_scale / (sqrtf(ss / p.true_vdim + p.eps) * (1.f + expf(-z)));
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int d = tid + k * DM_THREADS;
    if (d < V) p.out[b * p.o_ld + static_cast<long long>(h) * V + d] = __float2bfloat16(v[k] * f);
  }
}

// About one wave of CTAs, never finer than DD_MIN_SPLIT tokens.  Depends on host values only.
inline void diff_splits(int B, int H, int G, int max_ctx, int* nsplit, int* split_tokens) {
  const int groups = B * G * ((H / G + DD_HEADS - 1) / DD_HEADS);
  int ns = (max_ctx + DD_MIN_SPLIT - 1) / DD_MIN_SPLIT;
  int want = diff_decode_target_ctas() / (groups > 0 ? groups : 1);
  if (want < 1) want = 1;
  if (want > DD_MAX_SPLITS) want = DD_MAX_SPLITS;
  if (ns < 1) ns = 1;
  if (want < ns) ns = want;
  int st = ((max_ctx + ns - 1) / ns + 31) / 32 * 32;
  if (st < DD_MIN_SPLIT) st = DD_MIN_SPLIT;
  ns = (max_ctx + st - 1) / st;
  *nsplit = ns < 1 ? 1 : ns;
  *split_tokens = st;
}

template <int DP, int DV, int TOK>
int launch_dd(const DiffDecodeParams& p, int B, cudaStream_t st) {
  using Geo = DdGeo<DP, DV, TOK>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(diff_decode_kernel<DP, DV, TOK>, cudaFuncAttributeMaxDynamicSharedMemorySize, Geo::SMEM);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured = true;
  }
  const int yb = p.G * ((p.H / p.G + DD_HEADS - 1) / DD_HEADS);
  launch_k(diff_decode_kernel<DP, DV, TOK>, dim3(B, yb, p.nsplit), dim3(DD_WARPS * 32), Geo::SMEM, st, p);
  if (p.nsplit > 1) launch_k(diff_merge_kernel, dim3(B, p.H), dim3(DM_THREADS), 0, st, p);
  return launch_status();
}

}  // namespace gk

using namespace gk;

// ptrs: {proj, turns, pos, slots, cache};  dims: {rows, q_off, k_off, v_off, NQ, NK, D, VC, rot}
// All offsets and sizes are even; cached rows are NK * D + VC elements.
GK_EXPORT int gk_rotate_append(int is_fp32, void* const* ptrs, long long ld, const int* dims, float magnitude, void* stream) {
  if (dims[0] == 0) return 0;
  for (int i = 1; i < 9; ++i)
    if (dims[i] < 0 || (i != 4 && i != 5 && dims[i] % 2)) return -1;
  if (ld % 2 || dims[8] > dims[6] || dims[8] > DA_MAX_ROT) return -1;
  auto fill = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    RotateAppendParams<T> p;
    p.proj = static_cast<T*>(ptrs[0]); p.ld = ld;
    p.turns = static_cast<const float2*>(ptrs[1]);
    p.pos = static_cast<const int*>(ptrs[2]); p.slots = static_cast<const int*>(ptrs[3]);
    p.cache = static_cast<T*>(ptrs[4]);
    p.q_off = dims[1]; p.k_off = dims[2]; p.v_off = dims[3]; p.NQ = dims[4]; p.NK = dims[5]; p.D = dims[6]; p.VC = dims[7];
    p.rot = dims[8]; p.magnitude = magnitude;
    launch_k(rotate_append_kernel<T>, dim3(dims[0]), dim3(128), 0, reinterpret_cast<cudaStream_t>(stream), p);
    return launch_status();
  };
  return is_fp32 ? fill(static_cast<float*>(nullptr)) : fill(static_cast<__nv_bfloat16*>(nullptr));
}

// a [rows, H, maps, V] 32-bit (both maps, or with maps = 1 their difference) -> out rows o_ld apart, head h at h * V.
// ptrs: {a, gate, out, lam};  dims: {rows, H, maps, V, true_v};  floats: {out_scale, eps}
GK_EXPORT int gk_diff_combine(int is_fp32, int maps, void* const* ptrs, long long gate_ld, long long o_ld, const int* dims,
                              const float* floats, void* stream) {
  const int rows = dims[0], H = dims[1], V = dims[2], true_v = dims[3];
  if ((maps != 1 && maps != 2) || V < 1 || true_v < 1 || true_v > V) return -1;
  if (rows == 0) return 0;
  const dim3 grid(static_cast<unsigned>((static_cast<long long>(rows) * H + 3) / 4)), block(128);
  auto go = [&](auto* tag, auto m) {
    using T = std::remove_pointer_t<decltype(tag)>;
    launch_k(diff_finish_kernel<T, decltype(m)::value>, grid, block, 0, reinterpret_cast<cudaStream_t>(stream),
             static_cast<const float*>(ptrs[0]), static_cast<const T*>(ptrs[1]), gate_ld, static_cast<T*>(ptrs[2]), o_ld,
             static_cast<const float*>(ptrs[3]), rows, H, V, true_v, floats[0], floats[1]);
    return launch_status();
  };
  float* f = nullptr;
  __nv_bfloat16* h = nullptr;
  std::integral_constant<int, 1> one;
  std::integral_constant<int, 2> two;
  if (is_fp32) return maps == 1 ? go(f, one) : go(f, two);
  return maps == 1 ? go(h, one) : go(h, two);
}

GK_EXPORT void gk_diff_set_target_ctas(int n) { diff_decode_target_ctas() = n > 0 ? n : 444; }

// 1 when a kernel is built for maps of `dim` and values of `vdim` columns
GK_EXPORT int gk_diff_decode_supported(int dim, int vdim) { return dim >= 1 && dim <= 128 && vdim >= 1 && vdim <= 256; }

GK_EXPORT long long gk_diff_decode_scratch(int B, int H, int G, int vdim, int max_ctx) {
  int ns, st;
  diff_splits(B, H, G, max_ctx, &ns, &st);
  return ns > 1 ? static_cast<long long>(B) * H * 2 * ns * (vdim + 2) : 0;
}

// One new token per request; max_ctx bounds every ctx_len[b].
// ptrs: {proj, cache, tables, ctx_len, new_slots, turns, lam, out, scratch};  lds: {ld, o_ld}
// dims: {B, H, G, dim, vdim, true_vdim, rot, q_off, k_off, v_off, gate_off, row, block_size, max_blocks, max_ctx}
// floats: {scale, magnitude, out_scale, eps}
GK_EXPORT int gk_diff_decode(void* const* ptrs, const long long* lds, const int* dims, const float* floats, void* stream) {
  const int B = dims[0], H = dims[1], G = dims[2], dim = dims[3], vdim = dims[4];
  if (!gk_diff_decode_supported(dim, vdim) || G < 1 || H % G || dim % 8 || vdim % 8 || dims[6] % 2 || dims[6] > dim) return -1;
  if (lds[0] % 8 || dims[7] % 8 || dims[8] % 8 || dims[9] % 8 || dims[11] % 8 || dims[11] < G * (2 * dim + vdim)) return -1;
  if ((reinterpret_cast<uintptr_t>(ptrs[0]) | reinterpret_cast<uintptr_t>(ptrs[1])) & 15) return -1;
  if (B == 0) return 0;
  DiffDecodeParams p;
  p.proj = static_cast<const __nv_bfloat16*>(ptrs[0]); p.ld = lds[0];
  p.cache = static_cast<__nv_bfloat16*>(ptrs[1]);
  p.tables = static_cast<const int*>(ptrs[2]); p.ctx_len = static_cast<const int*>(ptrs[3]);
  p.new_slots = static_cast<const int*>(ptrs[4]);
  p.turns = static_cast<const float2*>(ptrs[5]); p.lam = static_cast<const float*>(ptrs[6]);
  p.out = static_cast<__nv_bfloat16*>(ptrs[7]); p.o_ld = lds[1];
  p.scratch = static_cast<float*>(ptrs[8]);
  p.H = H; p.G = G; p.dim = dim; p.vdim = vdim; p.true_vdim = dims[5]; p.rot = dims[6];
  p.q_off = dims[7]; p.k_off = dims[8]; p.v_off = dims[9]; p.gate_off = dims[10]; p.row = dims[11];
  p.block_size = dims[12]; p.max_blocks = dims[13];
  p.scale = floats[0]; p.magnitude = floats[1]; p.out_scale = floats[2]; p.eps = floats[3];
  diff_splits(B, H, G, dims[14], &p.nsplit, &p.split_tokens);
  if (p.nsplit > 1 && !p.scratch) return -2;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (dim <= 64) {
    if (vdim <= 64) return launch_dd<64, 64, 32>(p, B, st);
    return vdim <= 128 ? launch_dd<64, 128, 32>(p, B, st) : launch_dd<64, 256, 16>(p, B, st);
  }
  if (vdim <= 64) return launch_dd<128, 64, 16>(p, B, st);
  return vdim <= 128 ? launch_dd<128, 128, 16>(p, B, st) : launch_dd<128, 256, 16>(p, B, st);
}
