// Matrix memory (mLSTM) over prompt portions, 128 tokens at a time, on tcgen05 (see matrix_memory.cu for the recurrence
// and the state layout).  With b_t the running sum of the log forget gates inside a chunk, a_s = i_s - b_s and
// g_t = max(m_0, max_{s <= t} a_s), the running maximum is m_t = b_t + g_t and
//     o_t   = e^(m_0 - g_t) q_t S_0 + sum_{s <= t} e^(a_s - g_t) (q_t . k_s) v_s
//     S_end = e^(m_0 - g_end) S_0  + sum_s e^(a_s - g_end) k_s v_s^T          (n likewise, with 1 in place of v_s)
// so a chunk is four tensor-core products with 32-bit weights between them.  What the recurrence keeps in 32-bit and a
// product reads as bf16 - the decayed scores, the state, the weighted values - enters it as two bf16 terms (rounded
// value and remainder); the state itself stays in tensor memory in 32-bit from chunk to chunk.
//
// Retention (RET) is the case of constant gates, f = log(decay) and i = 0, without normaliser, maximum and denominator:
// a_s = -s log(decay), g_t = -t log(decay), and the state enters as if m_0 were log(decay).
//
// One CTA = one head of one portion and a slice of 64 value columns.  Keys of more than 128 dims are taken in halves.
//   warps 0-7   elementwise work: state -> operand, weighted values, decayed scores, output (lane quadrant = warp & 3,
//               column half = warp >> 2)
//   warp 8      TMA producer        warp 9  MMA issuer        warp 10  gates of the next chunk (scan over 128 tokens)
//
// The elementwise warps turn the state into the next chunk's operand before they wait for the current chunk's output, so
// the tensor core is fed while they finish it; inter-chunk outputs therefore alternate between two buffers.
//
// TMEM columns (512): scores [0,128), inter-chunk output 2 x 64 at 128, intra-chunk output [256,320), state 64 * NH at 320,
// normaliser 16 * NH at 448, q . n 2 x 16 at 480.
#include "ptx.cuh"
#include "host_utils.h"

namespace gk {

constexpr int MC_L = 128;          // tokens per chunk
constexpr int MC_DH = 128;         // key dims per half
constexpr int MC_SLICE = 64;       // value columns per CTA (= MM_SLICE of matrix_memory.cu)
constexpr int MC_THREADS = 352;
constexpr int MC_EW = 256;         // elementwise threads
constexpr float MC_LOG2E = 1.4426950408889634f;
constexpr uint32_t MC_T_S = 0, MC_T_OI = 128, MC_T_OA = 256, MC_T_ST = 320, MC_T_N = 448, MC_T_QN = 480;

struct McSmem {
  static constexpr int Q = 0;                    // [2 chunks of 64 dims][128 rows][128 B]
  static constexpr int K = Q + 32768;
  static constexpr int V = K + 32768;            // [128 rows][128 B]
  static constexpr int VW = V + 16384;           // weighted values: high terms, remainders
  static constexpr int P = VW + 32768;           // decayed scores: high terms [2 chunks of 64 keys], remainders
  static constexpr int ST = P + 65536;           // state operand: high terms [128 dims][128 B], remainders
  static constexpr int N = ST + 32768;           // normaliser operand: 16 rows (high, remainder, zeros) x 128 dims
  static constexpr int W = N + 4096;             // key weights: 16 rows (high, remainder, zeros) x 128 tokens
  static constexpr int GATES = W + 4096;         // [2][a 128 | g 128 | m 128 | m_0]
  static constexpr int GATE_FLOATS = 3 * MC_L + 4;
  static constexpr int RSUM = GATES + 2 * GATE_FLOATS * 4;   // [2][2][128] row sums of the scores
  static constexpr int BARS = RSUM + 2 * 2 * MC_L * 4;
  static constexpr int BYTES = BARS + 160;
};
static_assert(McSmem::BARS % 8 == 0 && McSmem::BYTES <= 232448, "fits the shared memory of one SM");

struct McParams {
  const float* gates;      // [rows, 2 * heads] projected gates without bias
  const float* gate_b;     // [2 * heads]
  const int* cu;           // [portions + 1]
  const int* first_pos;    // [portions] 0: the state starts at zero
  const int* slots;        // [portions]
  float* S;
  float* n;
  float* m;
  float* out;              // [rows, heads, vdim]
  int heads, dim, vdim, slices;
  float cap, q_scale;
  const float* decay;      // RET: [heads]; gates, gate_b, n and m are absent
  int* err;
};

__device__ __forceinline__ float mc_lo(float v, uint32_t hi_bits16) { return v - bf16_bits_to_float(static_cast<uint16_t>(hi_bits16)); }
// 8 values -> one 16-byte unit of rounded values and one of remainders
__device__ __forceinline__ void mc_split8(const float* v, uint4& hi, uint4& lo) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    h[e] = pack_bf16x2(v[2 * e], v[2 * e + 1]);
    l[e] = pack_bf16x2(mc_lo(v[2 * e], h[e] & 0xffff), mc_lo(v[2 * e + 1], h[e] >> 16));
  }
  hi = make_uint4(h[0], h[1], h[2], h[3]);
  lo = make_uint4(l[0], l[1], l[2], l[3]);
}
// element `e` of rows 0 (rounded) and 1 (remainder) of a 16-row K-major operand: 2048-byte chunks of 64 elements
__device__ __forceinline__ void mc_put_row01(uint8_t* base, int e, float v) {
  const uint32_t h = pack_bf16x2(v, 0.f) & 0xffff;
  const uint32_t l = pack_bf16x2(mc_lo(v, h), 0.f) & 0xffff;
  uint8_t* c = base + (e >> 6) * 2048 + (e & 7) * 2;
  const int u = (e & 63) >> 3;
  *reinterpret_cast<uint16_t*>(c + (u << 4)) = static_cast<uint16_t>(h);
  *reinterpret_cast<uint16_t*>(c + 128 + ((u ^ 1) << 4)) = static_cast<uint16_t>(l);
}

template <int NH, bool RET>
__global__ void __launch_bounds__(MC_THREADS, 1)
matrix_memory_chunk_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                           const __grid_constant__ CUtensorMap tmV, McParams p) {
  extern __shared__ __align__(1024) uint8_t smem[];
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + McSmem::BARS);
  uint64_t *qk_full = bars, *qk_empty = bars + 1, *v_full = bars + 2, *v_empty = bars + 3, *s_full = bars + 4,
           *sop_ready = bars + 5, *vw_ready = bars + 6, *p_ready = bars + 7, *upd_done = bars + 8, *o_done = bars + 9,
           *g_full = bars + 10 /* 2 */, *g_empty = bars + 12 /* 2 */;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + 14);
  float* gates_s = reinterpret_cast<float*>(smem + McSmem::GATES);
  float* rsum = reinterpret_cast<float*>(smem + McSmem::RSUM);

  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int head = blockIdx.x / p.slices, slice = blockIdx.x % p.slices, seg = blockIdx.y;
  const int r_beg = p.cu[seg], len = p.cu[seg + 1] - r_beg;
  const int slot = p.slots[seg];
  if (len <= 0 || slot < 0) return;          // uniform across the CTA, before any allocation
  if (smem_u32(smem) & 1023u) {
    if (tid == 0) atomicCAS(p.err, 0, ERR_WAIT_MISC);
    return;
  }
  const int chunks = (len + MC_L - 1) / MC_L;
  const bool fresh = p.first_pos[seg] == 0;
  const long long sh = static_cast<long long>(slot) * p.heads + head;
  float* ng = RET ? nullptr : p.n + (sh * p.slices + slice) * p.dim;
  float* mg = RET ? nullptr : p.m + sh * p.slices + slice;

  if (tid == 0) {
    mbar_init(qk_full, 1);
    mbar_init(qk_empty, 1);
    mbar_init(v_full, 1);
    mbar_init(v_empty, 1);
    mbar_init(s_full, 1);
    mbar_init(sop_ready, MC_EW);
    mbar_init(vw_ready, MC_EW);
    mbar_init(p_ready, MC_EW);
    mbar_init(upd_done, 1);
    mbar_init(o_done, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&g_full[i], 32);
      mbar_init(&g_empty[i], MC_EW);
    }
    fence_barrier_init();
    prefetch_tmap(&tmQ);
    prefetch_tmap(&tmK);
    prefetch_tmap(&tmV);
  }
  for (int i = tid; i < 8192 / 16; i += MC_THREADS)   // operand rows that stay zero (N and W are adjacent)
    *reinterpret_cast<uint4*>(smem + McSmem::N + i * 16) = make_uint4(0, 0, 0, 0);
  if (warp == 9) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(tmem_holder);

  if (warp == 8) {
    // ------------------------------------------------------------------ TMA producer
    bool ok = true;
    for (int c = 0; c < chunks && ok; ++c) {
      const int row = r_beg + c * MC_L;
      for (int h = 0; h < NH && ok; ++h) {
        const int it = c * NH + h;
        ok = mbar_wait(qk_empty, (it & 1) ^ 1, p.err, ERR_WAIT_EMPTY);
        if (!ok) break;
        if (lane == 0) {
          mbar_expect_tx(qk_full, 65536);
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            tma_load_3d(smem + McSmem::Q + x * 16384, &tmQ, qk_full, h * MC_DH + x * 64, head, row);
            tma_load_3d(smem + McSmem::K + x * 16384, &tmK, qk_full, h * MC_DH + x * 64, head, row);
          }
        }
        __syncwarp();
        if (h == 0) {
          ok = mbar_wait(v_empty, (c & 1) ^ 1, p.err, ERR_WAIT_EMPTY);
          if (!ok) break;
          if (lane == 0) {
            mbar_expect_tx(v_full, 16384);
            tma_load_3d(smem + McSmem::V, &tmV, v_full, slice * MC_SLICE, head, row);
          }
          __syncwarp();
        }
      }
    }
  } else if (warp == 9) {
    // ------------------------------------------------------------------ MMA issuer
    constexpr uint32_t id_s = make_idesc(128, 128, 1, 1, 0, 0);    // q k^T
    constexpr uint32_t id_o = make_idesc(128, 64, 1, 1, 0, 1);     // q S, P v: right operand stored [contraction][columns]
    constexpr uint32_t id_qn = make_idesc(128, 16, 1, 1, 0, 0);    // q . n
    constexpr uint32_t id_up = make_idesc(128, 64, 1, 1, 1, 1);    // k^T (w v)
    constexpr uint32_t id_un = make_idesc(128, 16, 1, 1, 1, 0);    // k^T w
    const uint32_t aQ = smem_u32(smem + McSmem::Q), aK = smem_u32(smem + McSmem::K), aV = smem_u32(smem + McSmem::V);
    const uint32_t aVW = smem_u32(smem + McSmem::VW), aP = smem_u32(smem + McSmem::P), aST = smem_u32(smem + McSmem::ST);
    const uint32_t aN = smem_u32(smem + McSmem::N), aW = smem_u32(smem + McSmem::W);
    bool ok = true;
    for (int c = 0; c < chunks && ok; ++c) {
      const uint32_t t_oi = tmem + MC_T_OI + (c & 1) * 64, t_qn = tmem + MC_T_QN + (c & 1) * 16;
      for (int h = 0; h < NH && ok; ++h) {
        const int it = c * NH + h;
        ok = mbar_wait(qk_full, it & 1, p.err, ERR_WAIT_FULL);
        if (!ok) break;
        tc_fence_after();
        if (lane == 0) {
#pragma unroll
          for (int k4 = 0; k4 < 8; ++k4) {
            const uint32_t o = (k4 >> 2) * 16384 + (k4 & 3) * 32;
            umma_f16(tmem + MC_T_S, make_smem_desc_sw128(aQ + o, 16, 1024), make_smem_desc_sw128(aK + o, 16, 1024), id_s,
                     (h > 0 || k4 > 0) ? 1u : 0u);
          }
          if (h == NH - 1) umma_commit(s_full);
        }
        __syncwarp();
        ok = mbar_wait(sop_ready, it & 1, p.err, ERR_WAIT_MISC);
        if (!ok) break;
        tc_fence_after();
        if (lane == 0) {
#pragma unroll
          for (int k4 = 0; k4 < 8; ++k4) {
            const uint64_t a = make_smem_desc_sw128(aQ + (k4 >> 2) * 16384 + (k4 & 3) * 32, 16, 1024);
            umma_f16(t_oi, a, make_smem_desc_sw128(aST + k4 * 2048, 16384, 1024), id_o, (h > 0 || k4 > 0) ? 1u : 0u);
            umma_f16(t_oi, a, make_smem_desc_sw128(aST + 16384 + k4 * 2048, 16384, 1024), id_o, 1u);
            if (!RET)
              umma_f16(t_qn, a, make_smem_desc_sw128(aN + (k4 >> 2) * 2048 + (k4 & 3) * 32, 16, 1024), id_qn,
                       (h > 0 || k4 > 0) ? 1u : 0u);
          }
        }
        __syncwarp();
        if (h == 0) {
          ok = mbar_wait(vw_ready, c & 1, p.err, ERR_WAIT_MISC);
          if (!ok) break;
          tc_fence_after();
        }
        if (lane == 0) {
#pragma unroll
          for (int k4 = 0; k4 < 8; ++k4) {
            const uint64_t a = make_smem_desc_sw128(aK + k4 * 2048, 16384, 1024);
            umma_f16(tmem + MC_T_ST + h * 64, a, make_smem_desc_sw128(aVW + k4 * 2048, 16384, 1024), id_up, 1u);
            umma_f16(tmem + MC_T_ST + h * 64, a, make_smem_desc_sw128(aVW + 16384 + k4 * 2048, 16384, 1024), id_up, 1u);
            if (!RET)
              umma_f16(tmem + MC_T_N + h * 16, a, make_smem_desc_sw128(aW + (k4 >> 2) * 2048 + (k4 & 3) * 32, 16, 1024), id_un, 1u);
          }
          umma_commit(upd_done);
          umma_commit(qk_empty);
        }
        __syncwarp();
      }
      if (!ok) break;
      ok = mbar_wait(p_ready, c & 1, p.err, ERR_WAIT_MISC);
      if (!ok) break;
      tc_fence_after();
      if (lane == 0) {
#pragma unroll
        for (int term = 0; term < 2; ++term) {
#pragma unroll
          for (int k4 = 0; k4 < 8; ++k4) {
            umma_f16(tmem + MC_T_OA, make_smem_desc_sw128(aP + term * 32768 + (k4 >> 2) * 16384 + (k4 & 3) * 32, 16, 1024),
                     make_smem_desc_sw128(aV + k4 * 2048, 16384, 1024), id_o, (term > 0 || k4 > 0) ? 1u : 0u);
          }
        }
        umma_commit(o_done);
        umma_commit(v_empty);
      }
      __syncwarp();
    }
  } else if (warp == 10) {
    // ------------------------------------------------------------------ gates: a, g, m of every token of a chunk
    const float bi = RET ? 0.f : p.gate_b[head], bf = RET ? 0.f : p.gate_b[p.heads + head];
    const float log_decay = RET ? fmaxf(logf(p.decay[head]), -80.f) : 0.f;
    float m0 = RET ? log_decay : fresh ? 0.f : *mg;
    bool ok = true;
    for (int c = 0; c < chunks; ++c) {
      const int buf = c & 1;
      ok = mbar_wait(&g_empty[buf], ((c >> 1) & 1) ^ 1, p.err, ERR_WAIT_EMPTY);
      if (!ok) break;
      float* gs = gates_s + buf * McSmem::GATE_FLOATS;
      if (RET) {
        const int last = len - c * MC_L - 1 < MC_L - 1 ? len - c * MC_L - 1 : MC_L - 1;   // newest token of the chunk
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int t = lane * 4 + j;
          gs[t] = t <= last ? -static_cast<float>(t) * log_decay : -1e30f;
          gs[MC_L + t] = -static_cast<float>(t < last ? t : last) * log_decay;
        }
        if (lane == 0) gs[3 * MC_L] = m0;
        mbar_arrive(&g_full[buf]);
        continue;
      }
      float gi[4], b[4];
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = c * MC_L + lane * 4 + j;
        float f = 0.f;
        gi[j] = -1e30f;                       // rows past the portion: no weight, no decay
        if (t < len) {
          const float* gr = p.gates + static_cast<long long>(r_beg + t) * 2 * p.heads + head;
          gi[j] = p.cap * tanhf((gr[0] + bi) / p.cap);
          const float z = p.cap * tanhf((gr[p.heads] + bf) / p.cap);
          f = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
        }
        sum += f;
        b[j] = sum;
      }
      float incl = sum;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffff, incl, o);
        if (lane >= o) incl += y;
      }
      float before = __shfl_up_sync(0xffffffff, incl, 1);
      if (lane == 0) before = 0.f;
      float a[4], mx = -1e30f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        b[j] += before;
        a[j] = gi[j] > -1e29f ? gi[j] - b[j] : -1e30f;
        mx = fmaxf(mx, a[j]);
      }
      float pm = mx;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffff, pm, o);
        if (lane >= o) pm = fmaxf(pm, y);
      }
      float g = __shfl_up_sync(0xffffffff, pm, 1);
      g = lane == 0 ? m0 : fmaxf(m0, g);
      float mt = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        g = fmaxf(g, a[j]);
        mt = b[j] + g;
        gs[lane * 4 + j] = a[j];
        gs[MC_L + lane * 4 + j] = g;
        gs[2 * MC_L + lane * 4 + j] = mt;
      }
      if (lane == 0) gs[3 * MC_L] = m0;
      m0 = __shfl_sync(0xffffffff, mt, 31);
      mbar_arrive(&g_full[buf]);
    }
    if (!RET && ok && lane == 0) *mg = m0;
  } else {
    // ------------------------------------------------------------------ elementwise warps
    const int quad = warp & 3, half = warp >> 2;
    const int r = quad * 32 + lane;                  // TMEM lane: key dim of the state, token of scores and outputs
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(quad * 32) << 16);
    const int col0 = slice * MC_SLICE + half * 32;   // first value column of this thread
    // state of the earlier steps -> tensor memory
#pragma unroll
    for (int h = 0; h < NH; ++h) {
      const int d = h * MC_DH + r;
      const bool have = !fresh && d < p.dim;
      uint32_t w[32];
      const float* src = p.S + (sh * p.dim + d) * p.vdim + col0;
#pragma unroll
      for (int j = 0; j < 32; j += 4) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (have && col0 + j < p.vdim) v = *reinterpret_cast<const float4*>(src + j);
        w[j] = __float_as_uint(v.x); w[j + 1] = __float_as_uint(v.y);
        w[j + 2] = __float_as_uint(v.z); w[j + 3] = __float_as_uint(v.w);
      }
      tmem_st32(lane_addr + MC_T_ST + h * 64 + half * 32, w);
      if (!RET && half == 0) {
        uint32_t nv[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) nv[j] = 0;
        if (have) nv[0] = __float_as_uint(ng[d]);
        tmem_st16(lane_addr + MC_T_N + h * 16, nv);
      }
    }
    tmem_st_wait();
    // state -> operand of q S (undecayed); its decayed value goes back to tensor memory for the update
    auto state_operand = [&](int c, int h) -> bool {
      const int it = c * NH + h;
      if (h == 0 && !mbar_wait(&g_full[c & 1], (c >> 1) & 1, p.err, ERR_WAIT_MISC)) return false;
      if (it > 0) {
        if (!mbar_wait(upd_done, (it - 1) & 1, p.err, ERR_WAIT_MISC)) return false;
        tc_fence_after();
      }
      const float* gs = gates_s + (c & 1) * McSmem::GATE_FLOATS;
      const float decay = ex2((gs[3 * MC_L] - gs[MC_L + MC_L - 1]) * MC_LOG2E);
      {
        uint32_t w[32];
        const uint32_t ta = lane_addr + MC_T_ST + h * 64 + half * 32;
        tmem_ld32(ta, w);
        tmem_ld_wait();
        uint8_t* dst = smem + McSmem::ST + r * 128;
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          float v[8];
          uint4 hi, lo;
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            v[e] = __uint_as_float(w[u * 8 + e]);
            w[u * 8 + e] = __float_as_uint(v[e] * decay);
          }
          mc_split8(v, hi, lo);
          const int o = ((half * 4 + u) ^ (r & 7)) << 4;
          *reinterpret_cast<uint4*>(dst + o) = hi;
          *reinterpret_cast<uint4*>(dst + 16384 + o) = lo;
        }
        tmem_st32(ta, w);
        if (!RET && half == 0) {
          uint32_t nv[16];
          tmem_ld16(lane_addr + MC_T_N + h * 16, nv);
          tmem_ld_wait();
          const float nn = __uint_as_float(nv[0]) + __uint_as_float(nv[1]);
          mc_put_row01(smem + McSmem::N, r, nn);
#pragma unroll
          for (int j = 0; j < 16; ++j) nv[j] = 0;
          nv[0] = __float_as_uint(nn * decay);
          tmem_st16(lane_addr + MC_T_N + h * 16, nv);
        }
        tmem_st_wait();
      }
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(sop_ready);
      return true;
    };
    // weighted values (token r, 32 columns) and key weights
    auto weighted_values = [&](int c) -> bool {
      if (!mbar_wait(v_full, c & 1, p.err, ERR_WAIT_FULL)) return false;
      const float* gs = gates_s + (c & 1) * McSmem::GATE_FLOATS;
      const float wt = ex2((gs[r] - gs[MC_L + MC_L - 1]) * MC_LOG2E);
      const uint8_t* src = smem + McSmem::V + r * 128;
      uint8_t* dst = smem + McSmem::VW + r * 128;
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int o = ((half * 4 + u) ^ (r & 7)) << 4;
        const uint4 x = *reinterpret_cast<const uint4*>(src + o);
        const uint32_t xs[4] = {x.x, x.y, x.z, x.w};
        float v[8];
        uint4 hi, lo;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          v[2 * e] = bf16_bits_to_float(static_cast<uint16_t>(xs[e] & 0xffff)) * wt;
          v[2 * e + 1] = bf16_bits_to_float(static_cast<uint16_t>(xs[e] >> 16)) * wt;
        }
        mc_split8(v, hi, lo);
        *reinterpret_cast<uint4*>(dst + o) = hi;
        *reinterpret_cast<uint4*>(dst + 16384 + o) = lo;
      }
      if (!RET && half == 0) mc_put_row01(smem + McSmem::W, r, wt);
      fence_proxy_async();
      mbar_arrive(vw_ready);
      return true;
    };
    // what a chunk needs from the elementwise warps behind its first state operand
    auto rest_of_operands = [&](int c) -> bool {
      bool fine = weighted_values(c);
#pragma unroll
      for (int h = 1; h < NH; ++h) fine = fine && state_operand(c, h);
      return fine;
    };
    const float log_qs = log2f(p.q_scale);
    bool ok = state_operand(0, 0) && rest_of_operands(0);
    for (int c = 0; c < chunks && ok; ++c) {
      const int buf = c & 1;
      const float* gs = gates_s + buf * McSmem::GATE_FLOATS;
      const float m0 = gs[3 * MC_L];
      // ---- decayed scores: token r against 64 keys
      const float g = gs[MC_L + r];
      ok = mbar_wait(s_full, c & 1, p.err, ERR_WAIT_TMEM_FULL);
      if (!ok) break;
      tc_fence_after();
      float rs = 0.f;
      uint8_t* prow = smem + McSmem::P + half * 16384 + r * 128;
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        uint32_t w[32];
        tmem_ld32(lane_addr + MC_T_S + half * 64 + x * 32, w);
        tmem_ld_wait();
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          float v[8];
          uint4 hi, lo;
          const int s0 = half * 64 + x * 32 + u * 8;
          const float4 a0 = *reinterpret_cast<const float4*>(gs + s0), a1 = *reinterpret_cast<const float4*>(gs + s0 + 4);
          const float av[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w};
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const float x2 = fmaf(av[e] - g, MC_LOG2E, log_qs);
            v[e] = __uint_as_float(w[u * 8 + e]) * ex2(s0 + e <= r ? x2 : -1e30f);
            if (!RET) rs += v[e];
          }
          mc_split8(v, hi, lo);
          const int o = ((x * 4 + u) ^ (r & 7)) << 4;
          *reinterpret_cast<uint4*>(prow + o) = hi;
          *reinterpret_cast<uint4*>(prow + 32768 + o) = lo;
        }
      }
      if (!RET) rsum[(buf * 2 + half) * MC_L + r] = rs;
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(p_ready);
      if (NH > 1 && c + 1 < chunks) {
        ok = state_operand(c + 1, 0);
        if (!ok) break;
      }
      // ---- output
      ok = mbar_wait(p_ready, c & 1, p.err, ERR_WAIT_MISC) && mbar_wait(o_done, c & 1, p.err, ERR_WAIT_TMEM_FULL);
      if (!ok) break;
      tc_fence_after();
      {
        const float inter = ex2((m0 - g) * MC_LOG2E) * p.q_scale;
        uint32_t qn[16], oi[32], oa[32];
        if (!RET) tmem_ld16(lane_addr + MC_T_QN + buf * 16, qn);
        tmem_ld32(lane_addr + MC_T_OI + buf * 64 + half * 32, oi);
        tmem_ld32(lane_addr + MC_T_OA + half * 32, oa);
        tmem_ld_wait();
        float inv = 1.f;
        if (!RET) {
          const float den = inter * (__uint_as_float(qn[0]) + __uint_as_float(qn[1])) + rsum[buf * 2 * MC_L + r] +
                            rsum[(buf * 2 + 1) * MC_L + r];
          inv = 1.f / (fmaxf(fabsf(den), ex2(-gs[2 * MC_L + r] * MC_LOG2E)) + 1e-6f);
        }
        // a warp's 32 x 32 outputs change hands in shared memory (the scores' buffer is free now), so that its stores
        // are whole 128-byte lines; 16-byte unit u of row r sits at unit u ^ (r & 7)
        uint8_t* stage = smem + McSmem::P + warp * 4096;
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          *reinterpret_cast<float4*>(stage + lane * 128 + ((u ^ (lane & 7)) << 4)) =
              make_float4((inter * __uint_as_float(oi[4 * u]) + __uint_as_float(oa[4 * u])) * inv,
                          (inter * __uint_as_float(oi[4 * u + 1]) + __uint_as_float(oa[4 * u + 1])) * inv,
                          (inter * __uint_as_float(oi[4 * u + 2]) + __uint_as_float(oa[4 * u + 2])) * inv,
                          (inter * __uint_as_float(oi[4 * u + 3]) + __uint_as_float(oa[4 * u + 3])) * inv);
        }
        __syncwarp();
        const int u = lane & 7, t0 = c * MC_L + quad * 32;
        float* dst = p.out + (static_cast<long long>(r_beg + t0) * p.heads + head) * p.vdim + col0 + u * 4;
#pragma unroll
        for (int x = 0; x < 8; ++x) {
          const int rr = x * 4 + (lane >> 3);
          const float4 v = *reinterpret_cast<const float4*>(stage + rr * 128 + ((u ^ (rr & 7)) << 4));
          if (t0 + rr < len && col0 + u * 4 < p.vdim)
            *reinterpret_cast<float4*>(dst + static_cast<long long>(rr) * p.heads * p.vdim) = v;
        }
        __syncwarp();
      }
      tc_fence_before();
      mbar_arrive(&g_empty[buf]);
      if (c + 1 < chunks) ok = (NH > 1 || state_operand(c + 1, 0)) && rest_of_operands(c + 1);
    }
    if (ok) {
      ok = mbar_wait(upd_done, (chunks * NH - 1) & 1, p.err, ERR_WAIT_MISC);
      if (ok) {
        tc_fence_after();
#pragma unroll
        for (int h = 0; h < NH; ++h) {
          const int d = h * MC_DH + r;
          uint32_t w[32], nv[16];
          tmem_ld32(lane_addr + MC_T_ST + h * 64 + half * 32, w);
          if (!RET) tmem_ld16(lane_addr + MC_T_N + h * 16, nv);
          tmem_ld_wait();
          if (d < p.dim) {
            float* dst = p.S + (sh * p.dim + d) * p.vdim + col0;
#pragma unroll
            for (int j = 0; j < 32; j += 4) {
              if (col0 + j < p.vdim) {
                *reinterpret_cast<float4*>(dst + j) = make_float4(__uint_as_float(w[j]), __uint_as_float(w[j + 1]),
                                                                  __uint_as_float(w[j + 2]), __uint_as_float(w[j + 3]));
              }
            }
            if (!RET && half == 0) ng[d] = __uint_as_float(nv[0]) + __uint_as_float(nv[1]);
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

template <int NH, bool RET>
int launch_mc(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const McParams& p, int portions,
              cudaStream_t st) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(matrix_memory_chunk_kernel<NH, RET>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         McSmem::BYTES);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured = true;
  }
  launch_k(matrix_memory_chunk_kernel<NH, RET>, dim3(p.heads * p.slices, portions), dim3(MC_THREADS), McSmem::BYTES, st, tq, tk,
           tv, p);
  return launch_status();
}

}  // namespace gk

using namespace gk;

// bf16 prompt portions, keys of at most 256 dims (a multiple of 8), values a multiple of 8 wide.
// ptrs: {proj, gates, gate_b, cu, first_pos, slots, S, n, m, out, err, decay}; decay (retention) replaces gates, gate_b, n, m
// dims: {portions, rows, q_off, k_off, v_off, heads, dim, vdim}
GK_EXPORT int gk_matrix_memory_chunk(void* const* ptrs, long long ld, const int* dims, float cap, float q_scale,
                                     void* stream) {
  const int n = dims[0], rows = dims[1], heads = dims[5], dim = dims[6], vdim = dims[7];
  if (n == 0) return 0;
  if (dim < 1 || dim > 2 * MC_DH || dim % 8 || vdim % 8 || ld % 8 || dims[2] % 8 || dims[3] % 8 || dims[4] % 8) return -1;
  const __nv_bfloat16* proj = static_cast<const __nv_bfloat16*>(ptrs[0]);
  if (reinterpret_cast<uintptr_t>(proj) & 15) return -1;
  CUtensorMap tq, tk, tv;
  if (make_tmap_3d(&tq, proj + dims[2], 2, rows, heads, dim, ld, dim, MC_L, 1, 64, true)) return -3;
  if (make_tmap_3d(&tk, proj + dims[3], 2, rows, heads, dim, ld, dim, MC_L, 1, 64, true)) return -4;
  if (make_tmap_3d(&tv, proj + dims[4], 2, rows, heads, vdim, ld, vdim, MC_L, 1, 64, true)) return -5;
  McParams p;
  p.gates = static_cast<const float*>(ptrs[1]);
  p.gate_b = static_cast<const float*>(ptrs[2]);
  p.cu = static_cast<const int*>(ptrs[3]);
  p.first_pos = static_cast<const int*>(ptrs[4]);
  p.slots = static_cast<const int*>(ptrs[5]);
  p.S = static_cast<float*>(ptrs[6]);
  p.n = static_cast<float*>(ptrs[7]);
  p.m = static_cast<float*>(ptrs[8]);
  p.out = static_cast<float*>(ptrs[9]);
  p.err = static_cast<int*>(ptrs[10]);
  p.decay = static_cast<const float*>(ptrs[11]);
  if (!p.decay && (!p.gates || !p.gate_b || !p.n || !p.m)) return -6;
  p.heads = heads; p.dim = dim; p.vdim = vdim; p.slices = (vdim + MC_SLICE - 1) / MC_SLICE;
  p.cap = cap; p.q_scale = q_scale;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (p.decay) return dim <= MC_DH ? launch_mc<1, true>(tq, tk, tv, p, n, st) : launch_mc<2, true>(tq, tk, tv, p, n, st);
  return dim <= MC_DH ? launch_mc<1, false>(tq, tk, tv, p, n, st) : launch_mc<2, false>(tq, tk, tv, p, n, st);
}
