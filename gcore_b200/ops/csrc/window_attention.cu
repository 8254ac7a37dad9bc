// Attention of decoders whose values are their keys: grouped-query softmax over a sliding window with a linear distance
// penalty, score = (q . k) * scale - slope_h * (i - j), on a paged cache that holds one row per (token, kv head).
//   * append_keys_kernel      copies the new keys of a packed projection into their cache slots;
//   * window_attn_kernel      any row (prompt portion or decoded token), any head size, 32-bit or bf16 storage, one warp
//                             per (row, head): the true 32-bit path and the sizes the tensor-core kernels do not cover.
//                             Keys and values may lie anywhere in a cached row and several keys may share a value;
//                             window, kept first positions, penalties, sink and output gate are optional and sigmoids may
//                             take the softmax's place, so absorbed latent attention, differential attention and attention
//                             with scored distances or sigmoid weights run on it too;
//   * shared_kv_decode_kernel one new token per request, bf16, head sizes 64 and 128: mma.sync tiles with the query heads
//                             of a group as rows (a group is far below the 64-row minimum of a tcgen05 instruction), KV
//                             splits, append of the new key fused in.
// Probabilities stay 32-bit: where they feed a tensor core they are split into two bf16 terms (high part + remainder).
// Prompt portions in bf16 run the tcgen05 kernel in window_prefill.cu.
#include "ptx.cuh"
#include "host_utils.h"
#include <cuda_bf16.h>
#include <float.h>
#include <type_traits>

namespace gk {

constexpr float WA_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float wa_f(float v) { return v; }
__device__ __forceinline__ float wa_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void wa_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void wa_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// proj rows [ld elements]; the keys are `n` contiguous elements at column k_off; slots[t] < 0: not stored.
// VT = 16-byte vector; n_vec vectors per row.
__global__ void append_keys_kernel(const uint4* __restrict__ proj, long long ld_vec, int off_vec, int n_vec,
                                   const int* __restrict__ slots, uint4* __restrict__ cache, int T) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
       i < static_cast<long long>(T) * n_vec; i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int t = static_cast<int>(i / n_vec), c = static_cast<int>(i - static_cast<long long>(t) * n_vec);
    const int s = slots[t];
    if (s >= 0) cache[static_cast<long long>(s) * n_vec + c] = proj[t * ld_vec + off_vec + c];
  }
}

constexpr int WA_WARPS = 8;
constexpr int WA_MAX_D = 1024;

template <typename T, typename O>
struct WindowAttnParams {
  const T* q;               // head h of a row at h * D
  long long q_ld;
  const T* cache;           // rows of `cache_row` elements: key kh at kh * D, value g at v_off + g * v_stride
  long long cache_row;
  int v_off, v_stride;
  const int *tables, *row_seq, *pos, *slots;   // slots[row] < 0 marks an inactive row (zero output)
  int max_blocks, block_size;
  const float* slopes;      // [H] or null
  const float* sinks;       // [H] or null: a logit that joins the softmax denominator
  const T* gate;            // one logit per row and head, rows gate_ld apart, or null
  long long gate_ld;
  const float *r1, *r2;     // [H] or null: r1 ln(1 + r2 distance) is taken off a score
  const float* head_bias;   // [H] or null: added to a score
  O* out;                   // head h of a row at h * DV, rows out_ld apart
  long long out_ld;
  int rows, H, G, maps;     // H query heads over G values, `maps` keys per value: head h takes key (g, h % maps)
  int D, DV, window, keep;  // window 0: unlimited; the first `keep` positions are seen whatever the window
  int sigmoid;              // weights are sigmoids of the scores, not normalised
  float scale, out_scale;
};

// One warp per (row, query head); DV <= 32 * NR.
template <typename T, typename O, int NR>
__global__ void __launch_bounds__(WA_WARPS * 32) window_attn_kernel(const WindowAttnParams<T, O> p) {
  extern __shared__ float wa_q[];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, D = p.D, DV = p.DV;
  const long long item = static_cast<long long>(blockIdx.x) * WA_WARPS + warp;
  if (item >= static_cast<long long>(p.rows) * p.H) return;
  const int row = static_cast<int>(item / p.H), h = static_cast<int>(item - static_cast<long long>(row) * p.H);
  O* orow = p.out + row * p.out_ld + static_cast<long long>(h) * DV;
  float acc[NR];
#pragma unroll
  for (int r = 0; r < NR; ++r) acc[r] = 0.f;
  float m = -FLT_MAX, l = 0.f;
  if (p.slots[row] >= 0) {
    if (p.sinks) {
      m = p.sinks[h];
      l = lane == 0 ? 1.f : 0.f;
    }
    float* sq = wa_q + warp * D;
    const T* qr = p.q + row * p.q_ld + static_cast<long long>(h) * D;
    for (int d = lane; d < D; d += 32) sq[d] = wa_f(qr[d]);
    __syncwarp();
    const int g = h / (p.H / p.G), i = p.pos[row];
    const long long k_off = static_cast<long long>(g * p.maps + h % p.maps) * D;
    const long long v_off = p.v_off + static_cast<long long>(g) * p.v_stride;
    const int* table = p.tables + static_cast<long long>(p.row_seq[row]) * p.max_blocks;
    const float slope = p.slopes ? p.slopes[h] : 0.f, bias = p.head_bias ? p.head_bias[h] : 0.f;
    const float r1 = p.r1 ? p.r1[h] : 0.f, r2 = p.r1 ? p.r2[h] : 0.f;
    int j0 = p.window > 0 ? i - p.window + 1 : 0;
    if (j0 < 0) j0 = 0;
    const int kept = p.keep < j0 ? p.keep : j0, count = kept + i + 1 - j0;   // places: kept positions, then the window
    for (int base = 0; base < count; base += 32) {
      const int place = base + lane, j = place < kept ? place : j0 + place - kept;
      const int nt = count - base < 32 ? count - base : 32;
      float s = -FLT_MAX;
      long long at = 0;
      if (place < count) {
        at = (static_cast<long long>(table[j / p.block_size]) * p.block_size + j % p.block_size) * p.cache_row;
        const T* kr = p.cache + at + k_off;
        float a = 0.f;
        for (int d = 0; d < D; ++d) a = fmaf(sq[d], wa_f(kr[d]), a);
        s = a * p.scale - slope * static_cast<float>(i - j) + bias;
        if (p.r1) s -= r1 * log1pf(r2 * static_cast<float>(i - j));
      }
      float mx = s;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffff, mx, o));
      const float mn = fmaxf(m, mx);
      float e;
      if (p.sigmoid) {
        e = place < count ? 1.f / (1.f + expf(-s)) : 0.f;
      } else {
        const float c = expf(m - mn);            // 0 on the first tile (m = -FLT_MAX)
        e = place < count ? expf(s - mn) : 0.f;
        m = mn;
        l = l * c + e;
#pragma unroll
        for (int r = 0; r < NR; ++r) acc[r] *= c;
      }
      for (int t = 0; t < nt; ++t) {
        const float pt = __shfl_sync(0xffffffff, e, t);
        const T* vr = p.cache + __shfl_sync(0xffffffff, at, t) + v_off;
#pragma unroll
        for (int r = 0; r < NR; ++r)
          if (r * 32 + lane < DV) acc[r] = fmaf(pt, wa_f(vr[r * 32 + lane]), acc[r]);
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffff, l, o);
  }
  float inv = p.sigmoid ? p.out_scale : l > 0.f ? p.out_scale / l : 0.f;
  if (p.gate) inv /= 1.f + expf(-wa_f(p.gate[row * p.gate_ld + h]));
#pragma unroll
  for (int r = 0; r < NR; ++r)
    if (r * 32 + lane < DV) wa_st(orow + r * 32 + lane, acc[r] * inv);
}

// ---------------------------------------------------------------------------------------------------- bf16 decode
__device__ __forceinline__ void wa_ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void wa_ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void wa_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t wa_pack(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float wa_rest(float v) { return v - __bfloat162float(__float2bfloat16(v)); }

constexpr int SD_WARPS = 4;
constexpr int SD_ROWS = 16;     // query heads per CTA (rows of an mma tile)
constexpr int SD_MIN_SPLIT = 128;
inline int& shared_decode_target_ctas() {
  static int n = 444;
  return n;
}

// grid (request, kv head x blocks of 16 query heads, split).  q / k: rows of the packed projection.
// ONE8: groups of up to 8 heads.  Rows 8-15 of the probability tile then carry the remainder terms of rows 0-7, so one
// product serves both terms, and the halves of the output tile are added at the end.
template <int D, bool ONE8>
__global__ void __launch_bounds__(SD_WARPS * 32, 3) shared_kv_decode_kernel(
    const __nv_bfloat16* __restrict__ proj, long long ld, int q_off, int k_off, __nv_bfloat16* __restrict__ cache,
    const int* __restrict__ tables, int max_blocks, const int* __restrict__ ctx_len, const int* __restrict__ new_slots,
    const float* __restrict__ slopes, __nv_bfloat16* __restrict__ out, float* __restrict__ scratch, int H, int G,
    int block_size, int window, float scale, int nsplit, int split_tokens) {
  constexpr int NC = D / 8;            // 16-byte chunks of a key row
  constexpr int RB = D * 2;            // bytes of a key row
  constexpr int SWZ = NC >= 16 ? 15 : 7;
  constexpr int TILE = 32 * RB;        // one warp tile: 32 tokens
  __shared__ __align__(16) uint8_t sq[SD_ROWS * RB];
  __shared__ float m_all[SD_WARPS][SD_ROWS], l_all[SD_WARPS][SD_ROWS];
  extern __shared__ __align__(16) uint8_t sd_dyn[];   // two key tiles per warp; the merge reuses them

  pdl_launch_dependents();
  pdl_wait();
  const int grp = H / G, hblocks = (grp + SD_ROWS - 1) / SD_ROWS;
  const int b = blockIdx.x, g = blockIdx.y / hblocks, hb = blockIdx.y % hblocks, split = blockIdx.z;
  const int h0 = g * grp + hb * SD_ROWS;                       // first query head of this CTA
  const int nh = grp - hb * SD_ROWS < SD_ROWS ? grp - hb * SD_ROWS : SD_ROWS;
  const int len = ctx_len[b];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int start = len > window ? len - window : 0;
  const int s0 = start + split * split_tokens;
  if (split > 0 && s0 >= len) return;                          // dead split: the combine kernel skips it
  const int s1 = s0 + split_tokens < len ? s0 + split_tokens : len;
  const int ntiles = s1 > s0 ? (s1 - s0 + 31) / 32 : 0;
  const __nv_bfloat16* prow = proj + b * ld;

  uint8_t* kt = sd_dyn + warp * 2 * TILE;
  const uint32_t kts = static_cast<uint32_t>(__cvta_generic_to_shared(kt));
  auto request_tile = [&](int t, int buf) {
    const int tok0 = s0 + t * 32;
    long long slot_l = 0;
    if (tok0 + lane < s1) {
      const int tok = tok0 + lane;
      slot_l = static_cast<long long>(tables[static_cast<long long>(b) * max_blocks + tok / block_size]) * block_size +
               tok % block_size;
    }
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int idx = i * 32 + lane, row = idx / NC, ch = idx % NC;
      const long long slot = __shfl_sync(0xffffffff, slot_l, row);
      const uint32_t nbytes = tok0 + row < s1 ? 16u : 0u;      // rows past the end are zero-filled
      const uint32_t dst = kts + buf * TILE + row * RB + ((ch ^ (row & SWZ)) << 4);
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst),
                   "l"(cache + (slot * G + g) * D + ch * 8), "r"(nbytes) : "memory");
    }
  };
  if (warp < ntiles) request_tile(warp, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");

  for (int i = tid; i < SD_ROWS * NC; i += SD_WARPS * 32) {
    const int r = i / NC, c = i % NC;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < nh) v = *reinterpret_cast<const uint4*>(prow + q_off + static_cast<long long>(h0 + r) * D + c * 8);
    *reinterpret_cast<uint4*>(sq + r * RB + ((c ^ (r & SWZ)) << 4)) = v;
  }
  __syncthreads();
  const bool appends = s1 == len && ntiles > 0;   // the newest position lies in the last tile of this split

  const int r0 = lane >> 2, cq = (lane & 3) * 2;
  float m_run[2] = {-FLT_MAX, -FLT_MAX}, l_run[2] = {0.f, 0.f};
  float o[NC][4];
#pragma unroll
  for (int j = 0; j < NC; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
  const float sl2 = scale * WA_LOG2E;
  const float slope[2] = {r0 < nh ? slopes[h0 + r0] * WA_LOG2E : 0.f, r0 + 8 < nh ? slopes[h0 + r0 + 8] * WA_LOG2E : 0.f};

  if (warp < ntiles) {
    uint32_t qa[D / 16][4];
    const uint32_t sqs = static_cast<uint32_t>(__cvta_generic_to_shared(sq));
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) {
      const int row = (lane & 7) + ((lane >> 3) & 1) * 8, ch = ks * 2 + (lane >> 4);
      wa_ldsm_x4(qa[ks], sqs + row * RB + ((ch ^ (row & SWZ)) << 4));
    }
    int buf = 0;
#pragma unroll 1
    for (int t = warp; t < ntiles; t += SD_WARPS, buf ^= 1) {
      if (t + SD_WARPS < ntiles) request_tile(t + SD_WARPS, buf ^ 1);
      asm volatile("cp.async.commit_group;" ::: "memory");
      asm volatile("cp.async.wait_group 1;" ::: "memory");
      __syncwarp();
      const int tok0 = s0 + t * 32;
      const int nt = s1 - tok0 < 32 ? s1 - tok0 : 32;
      uint8_t* tile = kt + buf * TILE;
      const uint32_t ts = kts + buf * TILE;
      if (appends && t == ntiles - 1) {
        // the cache row of the newest position is stale: take the key from the projection, and store it
        const int row = len - 1 - tok0;
        const int slot = new_slots[b];
        if (lane < NC) {
          const uint4 v = *reinterpret_cast<const uint4*>(prow + k_off + static_cast<long long>(g) * D + lane * 8);
          *reinterpret_cast<uint4*>(tile + row * RB + ((lane ^ (row & SWZ)) << 4)) = v;
          if (hb == 0 && slot >= 0)
            *reinterpret_cast<uint4*>(cache + (static_cast<long long>(slot) * G + g) * D + lane * 8) = v;
        }
        __syncwarp();
      }
      float sc[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll
        for (int kp = 0; kp < D / 32; ++kp) {
          uint32_t kb[4];
          const int row = j * 8 + (lane & 7), ch = kp * 4 + (lane >> 3);
          wa_ldsm_x4(kb, ts + row * RB + ((ch ^ (row & SWZ)) << 4));
          wa_mma(sc[j], qa[2 * kp], kb[0], kb[1]);
          wa_mma(sc[j], qa[2 * kp + 1], kb[2], kb[3]);
        }
      }
      constexpr int HV = ONE8 ? 1 : 2;     // row halves that hold scores
      float mx[2] = {-FLT_MAX, -FLT_MAX};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
#pragma unroll
        for (int e = 0; e < 2 * HV; ++e) {
          const int ti = j * 8 + cq + (e & 1), half = e >> 1;
          const float v = ti < nt ? sc[j][e] * sl2 - slope[half] * static_cast<float>(len - 1 - (tok0 + ti)) : -FLT_MAX;
          sc[j][e] = v;
          mx[half] = fmaxf(mx[half], v);
        }
      }
      float resc[2];
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
#pragma unroll
      for (int j = 0; j < NC; ++j) { o[j][0] *= resc[0]; o[j][1] *= resc[0]; o[j][2] *= resc[1]; o[j][3] *= resc[1]; }
      uint32_t ph[2][4], pl[2][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float pv[4];
#pragma unroll
        for (int e = 0; e < 2 * HV; ++e) {
          pv[e] = sc[j][e] == -FLT_MAX ? 0.f : ex2(sc[j][e] - m_run[e >> 1]);
          l_run[e >> 1] += pv[e];
        }
        ph[j >> 1][(j & 1) * 2] = wa_pack(pv[0], pv[1]);
        if (ONE8) {
          ph[j >> 1][(j & 1) * 2 + 1] = wa_pack(wa_rest(pv[0]), wa_rest(pv[1]));
        } else {
          ph[j >> 1][(j & 1) * 2 + 1] = wa_pack(pv[2], pv[3]);
          pl[j >> 1][(j & 1) * 2] = wa_pack(wa_rest(pv[0]), wa_rest(pv[1]));
          pl[j >> 1][(j & 1) * 2 + 1] = wa_pack(wa_rest(pv[2]), wa_rest(pv[3]));
        }
      }
#pragma unroll
      for (int kk = 0; kk < 2; ++kk) {
#pragma unroll
        for (int np = 0; np < NC / 2; ++np) {
          uint32_t vb[4];
          const int row = kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, ch = np * 2 + (lane >> 4);
          wa_ldsm_x4_t(vb, ts + row * RB + ((ch ^ (row & SWZ)) << 4));
          wa_mma(o[2 * np], ph[kk], vb[0], vb[1]);
          wa_mma(o[2 * np + 1], ph[kk], vb[2], vb[3]);
          if (!ONE8) {
            wa_mma(o[2 * np], pl[kk], vb[0], vb[1]);
            wa_mma(o[2 * np + 1], pl[kk], vb[2], vb[3]);
          }
        }
      }
      __syncwarp();   // every lane is done with the tile before it is refilled
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    l_run[u] += __shfl_xor_sync(0xffffffff, l_run[u], 1);
    l_run[u] += __shfl_xor_sync(0xffffffff, l_run[u], 2);
  }
  __syncthreads();
  float* o_all = reinterpret_cast<float*>(sd_dyn);   // [warp][16][D]
  if ((lane & 3) == 0) {
    m_all[warp][r0] = m_run[0]; l_all[warp][r0] = l_run[0];
    if (!ONE8) { m_all[warp][r0 + 8] = m_run[1]; l_all[warp][r0 + 8] = l_run[1]; }
  }
#pragma unroll
  for (int j = 0; j < NC; ++j) {
    if (ONE8) {
      *reinterpret_cast<float2*>(o_all + (warp * SD_ROWS + r0) * D + j * 8 + cq) =
          make_float2(o[j][0] + o[j][2], o[j][1] + o[j][3]);
    } else {
      *reinterpret_cast<float2*>(o_all + (warp * SD_ROWS + r0) * D + j * 8 + cq) = make_float2(o[j][0], o[j][1]);
      *reinterpret_cast<float2*>(o_all + (warp * SD_ROWS + r0 + 8) * D + j * 8 + cq) = make_float2(o[j][2], o[j][3]);
    }
  }
  __syncthreads();
  for (int i = tid; i < nh * D; i += SD_WARPS * 32) {
    const int r = i / D, d = i % D;
    float mm = -FLT_MAX;
#pragma unroll
    for (int w = 0; w < SD_WARPS; ++w) mm = fmaxf(mm, m_all[w][r]);
    float acc = 0.f, ls = 0.f;
#pragma unroll
    for (int w = 0; w < SD_WARPS; ++w) {
      const float f = m_all[w][r] == -FLT_MAX ? 0.f : ex2(m_all[w][r] - mm);
      acc += o_all[(w * SD_ROWS + r) * D + d] * f;
      ls += l_all[w][r] * f;
    }
    const long long hh = static_cast<long long>(b) * H + h0 + r;
    if (nsplit == 1) {
      out[hh * D + d] = __float2bfloat16(ls > 0.f ? acc / ls : 0.f);
    } else {
      float* dst = scratch + (hh * nsplit + split) * (D + 2);
      dst[d] = acc;
      if (d == 0) { dst[D] = mm; dst[D + 1] = ls; }
    }
  }
}

template <int D>
__global__ void shared_kv_combine_kernel(const float* __restrict__ scratch, const int* __restrict__ ctx_len, int window,
                                         __nv_bfloat16* __restrict__ out, int H, int nsplit_total, int split_tokens) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y, d = threadIdx.x;
  const float* base = scratch + (static_cast<long long>(b) * H + h) * nsplit_total * (D + 2);
  const int span = ctx_len[b] < window ? ctx_len[b] : window;
  int ns = (span + split_tokens - 1) / split_tokens;
  ns = ns < 1 ? 1 : (ns > nsplit_total ? nsplit_total : ns);
  float m = -FLT_MAX;
  for (int s = 0; s < ns; ++s) m = fmaxf(m, base[s * (D + 2) + D]);
  float l = 0.f, acc = 0.f;
  for (int s = 0; s < ns; ++s) {
    const float ms = base[s * (D + 2) + D];
    const float w = ms == -FLT_MAX ? 0.f : ex2(ms - m);
    l += base[s * (D + 2) + D + 1] * w;
    acc += base[s * (D + 2) + d] * w;
  }
  out[(static_cast<long long>(b) * H + h) * D + d] = __float2bfloat16(l > 0.f ? acc / l : 0.f);
}

template <typename T, typename O>
int launch_window_attn(const WindowAttnParams<T, O>& p, cudaStream_t st) {
  const long long items = static_cast<long long>(p.rows) * p.H;
  const dim3 grid(static_cast<unsigned>((items + WA_WARPS - 1) / WA_WARPS)), block(WA_WARPS * 32);
  const size_t smem = WA_WARPS * p.D * sizeof(float);
  if (p.DV <= 128) launch_k(window_attn_kernel<T, O, 4>, grid, block, smem, st, p);
  else if (p.DV <= 512) launch_k(window_attn_kernel<T, O, 16>, grid, block, smem, st, p);
  else launch_k(window_attn_kernel<T, O, 32>, grid, block, smem, st, p);
  return launch_status();
}

// Splits the window so that the grid about fills the GPU once, never finer than 128 tokens.
inline void shared_decode_splits(int B, int yblocks, int span, int* nsplit, int* split_tokens) {
  int ns = (span + SD_MIN_SPLIT - 1) / SD_MIN_SPLIT;
  int want = shared_decode_target_ctas() / (B * yblocks > 0 ? B * yblocks : 1);
  if (want < 1) want = 1;
  if (ns < 1) ns = 1;
  if (want < ns) ns = want;
  int st = ((span + ns - 1) / ns + 31) / 32 * 32;
  if (st < SD_MIN_SPLIT) st = SD_MIN_SPLIT;
  ns = (span + st - 1) / st;
  *nsplit = ns < 1 ? 1 : ns;
  *split_tokens = st;
}

template <int D, bool ONE8>
int launch_shared_decode_impl(const void* proj, long long ld, int q_off, int k_off, void* cache, const int* tables,
                         int max_blocks, const int* ctx, const int* new_slots, const float* slopes, void* out,
                         float* scratch, int B, int H, int G, int block_size, int window, int max_ctx, float scale,
                         cudaStream_t st) {
  constexpr int SMEM = SD_WARPS * 2 * 32 * D * 2;
  static_assert(SMEM >= SD_WARPS * SD_ROWS * D * 4, "the merge fits the key tiles");
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(shared_kv_decode_kernel<D, ONE8>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    configured = true;
  }
  const int grp = H / G, yb = G * ((grp + SD_ROWS - 1) / SD_ROWS);
  int nsplit, split_tokens;
  shared_decode_splits(B, yb, window < max_ctx ? window : max_ctx, &nsplit, &split_tokens);
  if (nsplit > 1 && !scratch) return -2;
  launch_k(shared_kv_decode_kernel<D, ONE8>, dim3(B, yb, nsplit), dim3(SD_WARPS * 32), SMEM, st,
           static_cast<const __nv_bfloat16*>(proj), ld, q_off, k_off, static_cast<__nv_bfloat16*>(cache), tables,
           max_blocks, ctx, new_slots, slopes, static_cast<__nv_bfloat16*>(out), scratch, H, G, block_size, window, scale,
           nsplit, split_tokens);
  if (nsplit > 1)
    launch_k(shared_kv_combine_kernel<D>, dim3(B, H), dim3(D), 0, st, static_cast<const float*>(scratch), ctx, window,
             static_cast<__nv_bfloat16*>(out), H, nsplit, split_tokens);
  return launch_status();
}

template <int D, typename... A>
int launch_shared_decode(bool one8, A... a) {
  return one8 ? launch_shared_decode_impl<D, true>(a...) : launch_shared_decode_impl<D, false>(a...);
}

}  // namespace gk

using namespace gk;

// Keys: `n_bytes` contiguous bytes per row at byte offset `off` of projection rows `ld_bytes` apart (all multiples of 16).
GK_EXPORT int gk_append_keys(const void* proj, long long ld_bytes, long long off, int n_bytes, const int* slots,
                             void* cache, int T, void* stream) {
  if (ld_bytes % 16 || off % 16 || n_bytes % 16 || (reinterpret_cast<uintptr_t>(proj) & 15)) return -1;
  if (T == 0) return 0;
  const long long n = static_cast<long long>(T) * (n_bytes / 16);
  long long blocks = (n + 255) / 256;
  if (blocks > sm_count() * 8) blocks = sm_count() * 8;
  launch_k(append_keys_kernel, dim3(static_cast<unsigned>(blocks)), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream),
           static_cast<const uint4*>(proj), ld_bytes / 16, static_cast<int>(off / 16), n_bytes / 16, slots,
           static_cast<uint4*>(cache), T);
  return launch_status();
}

// ptrs: {q, cache, tables, row_seq, pos, slots, slopes, gate, out, sinks, r1, r2, head_bias}; slopes, gate and all behind out:
// or null;  lds: {q_ld, gate_ld, cache_row, out_ld};  window 0: unlimited;  out_fp32: 32-bit output of bf16 rows
// dims: {rows, H, G, maps, D, DV, v_off, v_stride, window, block_size, max_blocks, keep, sigmoid};  floats: {scale, out_scale}
GK_EXPORT int gk_window_attn(int is_fp32, int out_fp32, void* const* ptrs, const long long* lds, const int* dims,
                             const float* floats, void* stream) {
  const int H = dims[1], G = dims[2], maps = dims[3], D = dims[4], DV = dims[5];
  if (G < 1 || H % G || maps < 1 || (H / G) % maps || D < 1 || D > WA_MAX_D || DV < 1 || DV > WA_MAX_D || dims[8] < 0)
    return -1;
  if (dims[11] < 0 || lds[3] < static_cast<long long>(H) * DV || (ptrs[10] != nullptr) != (ptrs[11] != nullptr) ||
      (dims[12] && ptrs[9]))
    return -1;
  if (static_cast<long long>(G) * maps * D > lds[2] || dims[6] + static_cast<long long>(G - 1) * dims[7] + DV > lds[2])
    return -1;
  if (dims[0] == 0) return 0;
  auto fill = [&](auto* tag, auto* otag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    using O = std::remove_pointer_t<decltype(otag)>;
    WindowAttnParams<T, O> p;
    p.q = static_cast<const T*>(ptrs[0]); p.q_ld = lds[0];
    p.cache = static_cast<const T*>(ptrs[1]); p.cache_row = lds[2];
    p.v_off = dims[6]; p.v_stride = dims[7];
    p.tables = static_cast<const int*>(ptrs[2]); p.row_seq = static_cast<const int*>(ptrs[3]);
    p.pos = static_cast<const int*>(ptrs[4]); p.slots = static_cast<const int*>(ptrs[5]);
    p.max_blocks = dims[10]; p.block_size = dims[9];
    p.slopes = static_cast<const float*>(ptrs[6]); p.sinks = static_cast<const float*>(ptrs[9]);
    p.gate = static_cast<const T*>(ptrs[7]); p.gate_ld = lds[1];
    p.out = static_cast<O*>(ptrs[8]);
    p.rows = dims[0]; p.H = H; p.G = G; p.maps = maps; p.D = D; p.DV = DV; p.window = dims[8];
    p.r1 = static_cast<const float*>(ptrs[10]); p.r2 = static_cast<const float*>(ptrs[11]);
    p.head_bias = static_cast<const float*>(ptrs[12]); p.out_ld = lds[3];
    p.keep = dims[11]; p.sigmoid = dims[12]; p.scale = floats[0]; p.out_scale = floats[1];
    return launch_window_attn(p, reinterpret_cast<cudaStream_t>(stream));
  };
  float* f = nullptr;
  __nv_bfloat16* h = nullptr;
  return is_fp32 ? fill(f, f) : out_fp32 ? fill(h, f) : fill(h, h);
}

GK_EXPORT void gk_shared_decode_set_target_ctas(int n) { shared_decode_target_ctas() = n > 0 ? n : 444; }

// Scratch floats gk_shared_kv_decode may need (any split count at most ceil(span / 128)).
GK_EXPORT long long gk_shared_kv_decode_scratch(int B, int H, int D, int span) {
  return static_cast<long long>(B) * H * ((span + SD_MIN_SPLIT - 1) / SD_MIN_SPLIT + 1) * (D + 2);
}

// One new token per request (bf16, D = 64 or 128).  ctx[b] counts the new token; 0 = inactive row (zero output).
// dims: {B, H, G, D, window, block_size, max_blocks, max_ctx, q_off, k_off}
GK_EXPORT int gk_shared_kv_decode(const void* proj, long long ld, void* cache, const int* tables, const int* ctx,
                                  const int* new_slots, const float* slopes, void* out, float* scratch, const int* dims,
                                  float scale, void* stream) {
  const int B = dims[0], H = dims[1], G = dims[2], D = dims[3];
  if (H % G || dims[4] < 1 || ld % 8 || dims[8] % 8 || dims[9] % 8) return -1;
  if (B == 0) return 0;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (D == 64)
    return launch_shared_decode<64>(H / G <= 8, proj, ld, dims[8], dims[9], cache, tables, dims[6], ctx, new_slots, slopes, out,
                                    scratch, B, H, G, dims[5], dims[4], dims[7], scale, st);
  if (D == 128)
    return launch_shared_decode<128>(H / G <= 8, proj, ld, dims[8], dims[9], cache, tables, dims[6], ctx, new_slots, slopes, out,
                                     scratch, B, H, G, dims[5], dims[4], dims[7], scale, st);
  return -4;
}
