// Matrix memory (mLSTM): per head S_t = e^(f + m - m') S + e^(i - m') k v^T, n likewise with k alone, running maximum
// m' = max(f + m, i), output S^T q / (max(|n . q|, e^-m') + 1e-6).  All of it is 32-bit; q, k, v arrive in the storage
// type of the projection.
//   * matrix_memory_scan_kernel  token by token with the state slice in registers: decoding (one token per request, the
//                                gate projections fused in) and the true 32-bit path for prompt portions;
//                                One token per request with at most 8 slices: the slices of a head form a cluster, share
//                                their sums of squares through distributed shared memory and write the finished output;
//   * memory_output_kernel       per-head RMS norm, gain and sigmoid output gate behind every other case.
// bf16 prompt portions run the chunkwise kernel in matrix_memory_chunk.cu.
//
// Retention is the same recurrence with constant gates and without normaliser and maximum: S_t = decay S + k v^T, output
// S^T q, normed per head without a gain and gated by a silu, or normed over all heads together with a gain and gated by a
// sigmoid (memory_output_joint_kernel).  The RET instances of the kernels compute it.  The scan can rotate queries and keys, or
// apply a silu to queries, keys and values, as it reads them (in 32-bit).
//
// State layout per layer run: S [slots, heads, dim, vdim], n [slots, heads, slices, dim], m [slots, heads, slices]: a head's
// value columns are cut into slices of 64 that different CTAs own, and each keeps its own copy of n and m, so no CTA
// reads what another one writes.
#include "host_utils.h"
#include "rotary.cuh"
#include "row_ops.cuh"
#include <cuda_bf16.h>
#include <type_traits>

namespace gk {

constexpr int MM_SLICE = 64;
constexpr int MM_THREADS = 256;
constexpr int MM_MAX_ROT = 512;

__device__ __forceinline__ float mm_f(float v) { return v; }
__device__ __forceinline__ float mm_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float4 mm_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 mm_ld4(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void mm_st4(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void mm_st4(__nv_bfloat16* p, float a, float b, float c, float d) {
  __nv_bfloat162 x = __floats2bfloat162_rn(a, b), y = __floats2bfloat162_rn(c, d);
  uint2 r;
  r.x = *reinterpret_cast<uint32_t*>(&x);
  r.y = *reinterpret_cast<uint32_t*>(&y);
  *reinterpret_cast<uint2*>(p) = r;
}
__device__ __forceinline__ float mm_logsigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

template <typename T>
struct ScanParams {
  const T* proj;           // packed projection rows
  long long ld;
  int q_off, k_off, v_off;
  const T* h;              // [rows, width] mixer input, with gate_w: the gate projections are computed here
  const T* gate_w;         // [2 * heads, width]: input gates, then forget gates
  const float* gates;      // or: [rows, 2 * heads] projected gates without bias
  const float* gate_b;     // [2 * heads]
  const int* cu;           // [n + 1] first row of every segment, or null: one row per segment
  const int* first_pos;    // position of every segment's first token (0: the state starts at zero)
  const int* slots;        // state slot per segment; negative: inactive (zero output, no state touched)
  float* S;
  float* n;
  float* m;
  float* out;              // [rows, heads, vdim] 32-bit (unless the output is finished here)
  T* y;                    // FINISH: [rows, heads * vdim] normed and gated output
  const float* gain;       // FINISH: [heads * vdim]
  long long y_ld;          // FINISH: elements between rows of y
  int g_off, vdim_true;    // FINISH
  float eps;               // FINISH
  const float* decay;      // RET: [heads]; gates, n and m are absent
  const float2* turns;     // RET: [rot / 2] turns per position (value, remainder): leading dimensions rotated, neighbours paired
  int rot, act;            // RET: act: silu on queries, keys and values
  int width, heads, dim, vdim, slices;
  float cap, q_scale, out_scale;
};

__device__ __forceinline__ void mm_cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void mm_cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ void mm_store_remote(const float* local, uint32_t cta, float v) {
  const uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(local));
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(a), "r"(cta));
  asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(r), "f"(v) : "memory");
}
__device__ __forceinline__ void mm_st1(float* p, float v) { *p = v; }
__device__ __forceinline__ void mm_st1(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ float mm_gate(float g, bool silu) { return (silu ? g : 1.f) / (1.f + expf(-g)); }
__device__ __forceinline__ float mm_silu(float g) { return g / (1.f + expf(-g)); }

// grid (heads * slices, segments).  Thread (warp w, lane): rows rg, rg + 16, ... with rg = 2 w + lane / 16; columns
// 4 * (lane % 16) .. + 3 of the slice.  R = rows per thread.
template <typename T, int R, bool FINISH, bool RET>
__global__ void __launch_bounds__(MM_THREADS, R <= 8 ? 3 : R <= 16 ? 2 : 1) matrix_memory_scan_kernel(const ScanParams<T> p) {
  __shared__ float sq[2][16 * R], sk[2][16 * R];
  __shared__ float red[2][8][MM_SLICE + 4];
  __shared__ float gred[2][8];
  __shared__ float peer_ss[8];      // FINISH: sum of squares of every slice of the head
  __shared__ float warp_ss[2];
  __shared__ float s_cos[RET ? 8 * R : 1], s_sin[RET ? 8 * R : 1];   // rot / 2 of them
  pdl_launch_dependents();
  pdl_wait();
  const int head = blockIdx.x / p.slices, slice = blockIdx.x % p.slices, seg = blockIdx.y;
  const int r_beg = p.cu ? p.cu[seg] : seg, r_end = p.cu ? p.cu[seg + 1] : seg + 1;
  const int slot = p.slots[seg];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rg = warp * 2 + (lane >> 4), c0 = (lane & 15) * 4;
  const int col = slice * MM_SLICE + c0;                 // vdim is a multiple of 4
  const bool live = col < p.vdim;
  if (slot < 0) {
    for (int r = r_beg; r < r_end; ++r)
      if (tid < MM_SLICE && slice * MM_SLICE + tid < p.vdim) {
        const long long at = (static_cast<long long>(r) * p.heads + head) * p.vdim + slice * MM_SLICE + tid;
        if (FINISH) mm_st1(p.y + r * p.y_ld + static_cast<long long>(head) * p.vdim + slice * MM_SLICE + tid, 0.f);
        else p.out[at] = 0.f;
      }
    return;      // uniform over the slices of the head
  }
  if (FINISH) mm_cluster_arrive();
  const long long sh = static_cast<long long>(slot) * p.heads + head;
  float* Sg = p.S + sh * p.dim * p.vdim + col;
  float* ng = RET ? nullptr : p.n + (sh * p.slices + slice) * p.dim;
  float* mg = RET ? nullptr : p.m + sh * p.slices + slice;
  const bool fresh = p.first_pos[seg] == 0;
  float4 S[R];
  float n[R];
  float m = RET || fresh ? 0.f : *mg;
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int r = rg + 16 * j;
    S[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    n[j] = 0.f;
    if (!fresh && r < p.dim) {
      if (live) S[j] = *reinterpret_cast<const float4*>(Sg + static_cast<long long>(r) * p.vdim);
      if (!RET) n[j] = ng[r];
    }
  }
  auto store_state = [&]() {
#pragma unroll
    for (int j = 0; j < R; ++j) {
      const int r = rg + 16 * j;
      if (r < p.dim) {
        if (live) *reinterpret_cast<float4*>(Sg + static_cast<long long>(r) * p.vdim) = S[j];
        if (!RET && c0 == 0) ng[r] = n[j];
      }
    }
    if (!RET && tid == 0) *mg = m;
  };
  const float bi = RET ? 0.f : p.gate_b[head], bf = RET ? 0.f : p.gate_b[p.heads + head];
  const float decay = RET ? p.decay[head] : 0.f;
  for (int row = r_beg, it = 0; row < r_end; ++row, ++it) {
    const int buf = it & 1;
    const T* pr = p.proj + row * p.ld;
    const T *qr = pr + p.q_off + static_cast<long long>(head) * p.dim, *kr = pr + p.k_off + static_cast<long long>(head) * p.dim;
    if (RET && p.rot) {
      __syncthreads();       // the row before has read its angles
      for (int i = tid; i < p.rot >> 1; i += MM_THREADS) rotation_at(p.first_pos[seg] + it, p.turns[i], &s_sin[i], &s_cos[i]);
      __syncthreads();
    }
    for (int d = tid; d < 16 * R; d += MM_THREADS) {
      float q = d < p.dim ? mm_f(qr[d]) : 0.f, k = d < p.dim ? mm_f(kr[d]) : 0.f;
      if (RET && d < p.rot) {
        const float c = s_cos[d >> 1], s = d & 1 ? s_sin[d >> 1] : -s_sin[d >> 1];
        q = q * c + mm_f(qr[d ^ 1]) * s;
        k = k * c + mm_f(kr[d ^ 1]) * s;
      }
      if (RET && p.act) {
        q = mm_silu(q);
        k = mm_silu(k);
      }
      sq[buf][d] = q * p.q_scale;
      sk[buf][d] = k;
    }
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live) v = mm_ld4(pr + p.v_off + static_cast<long long>(head) * p.vdim + col);
    if (RET && p.act) v = make_float4(mm_silu(v.x), mm_silu(v.y), mm_silu(v.z), mm_silu(v.w));
    float gi = 0.f, gf = 0.f;
    if (RET) {
    } else if (p.gates) {
      gi = p.gates[static_cast<long long>(row) * 2 * p.heads + head];
      gf = p.gates[static_cast<long long>(row) * 2 * p.heads + p.heads + head];
    } else {
      const T* hr = p.h + static_cast<long long>(row) * p.width;
      const T* wi = p.gate_w + static_cast<long long>(head) * p.width;
      const T* wf = p.gate_w + static_cast<long long>(p.heads + head) * p.width;
      float a = 0.f, b = 0.f;
      for (int d = tid * 4; d < p.width; d += MM_THREADS * 4) {
        const float4 x = mm_ld4(hr + d), u = mm_ld4(wi + d), w = mm_ld4(wf + d);
        a += x.x * u.x + x.y * u.y + x.z * u.z + x.w * u.w;
        b += x.x * w.x + x.y * w.y + x.z * w.z + x.w * w.w;
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        a += __shfl_xor_sync(0xffffffff, a, o);
        b += __shfl_xor_sync(0xffffffff, b, o);
      }
      if (lane == 0) { gred[0][warp] = a; gred[1][warp] = b; }
      __syncthreads();
      gi = gf = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) { gi += gred[0][w]; gf += gred[1][w]; }
    }
    __syncthreads();
    float keep = decay, put = 1.f;
    if (!RET) {
      gi = p.cap * tanhf((gi + bi) / p.cap);
      gf = mm_logsigmoid(p.cap * tanhf((gf + bf) / p.cap));
      const float mn = fmaxf(gf + m, gi);
      keep = expf(gf + m - mn);
      put = expf(gi - mn);
      m = mn;
    }
    float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f, nq = 0.f;
#pragma unroll
    for (int j = 0; j < R; ++j) {
      const float q = sq[buf][rg + 16 * j], k = sk[buf][rg + 16 * j] * put;
      if (!RET) {
        n[j] = keep * n[j] + k;
        nq += n[j] * q;
      }
      S[j].x = keep * S[j].x + k * v.x; a0 += S[j].x * q;
      S[j].y = keep * S[j].y + k * v.y; a1 += S[j].y * q;
      S[j].z = keep * S[j].z + k * v.z; a2 += S[j].z * q;
      S[j].w = keep * S[j].w + k * v.w; a3 += S[j].w * q;
    }
    if (FINISH) store_state();   // on its way while the slices exchange their sums
    a0 += __shfl_xor_sync(0xffffffff, a0, 16);
    a1 += __shfl_xor_sync(0xffffffff, a1, 16);
    a2 += __shfl_xor_sync(0xffffffff, a2, 16);
    a3 += __shfl_xor_sync(0xffffffff, a3, 16);
    if (!RET) nq += __shfl_xor_sync(0xffffffff, nq, 16);
    if (lane < 16) {
      *reinterpret_cast<float4*>(&red[buf][warp][c0]) = make_float4(a0, a1, a2, a3);
      if (!RET && lane == 0) red[buf][warp][MM_SLICE] = nq;
    }
    __syncthreads();
    float o = 0.f;
    const int oc = slice * MM_SLICE + tid;
    const bool mine = tid < MM_SLICE && oc < p.vdim;
    if (mine) {
      float d = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        o += red[buf][w][tid];
        if (!RET) d += red[buf][w][MM_SLICE];
      }
      if (!RET) o = o / (fmaxf(fabsf(d), expf(-m)) + 1e-6f);
      if (!FINISH) p.out[(static_cast<long long>(row) * p.heads + head) * p.vdim + oc] = o;
    }
    if (FINISH) {   // one row per segment
      float gate = 0.f, gain = 1.f;
      if (mine) {
        gate = mm_f(pr[p.g_off + static_cast<long long>(head) * p.vdim + oc]);
        if (!RET) gain = p.gain[head * p.vdim + oc];
      }
      if (warp < 2) {
        float ss = o * o;
#pragma unroll
        for (int x = 16; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffff, ss, x);
        if (lane == 0) warp_ss[warp] = ss;
      }
      __syncthreads();
      mm_cluster_wait();                       // every slice has started: its shared memory may be written
      if (tid < p.slices) mm_store_remote(&peer_ss[slice], tid, warp_ss[0] + warp_ss[1]);
      mm_cluster_arrive();
      mm_cluster_wait();
      if (mine) {
        float ss = 0.f;
        for (int x = 0; x < p.slices; ++x) ss += peer_ss[x];
        const float r = 1.f / sqrtf(ss / p.vdim_true + p.eps);
        mm_st1(p.y + row * p.y_ld + static_cast<long long>(head) * p.vdim + oc,
               o * r * gain * mm_gate(gate, RET) * p.out_scale);
      }
    }
  }
  if (!FINISH && r_end > r_beg) store_state();
}

// y = o / rms(o over the head's true size) * gain * sigmoid(g), or without a gain: ... * silu(g).  One warp per
// (row, head).
template <typename T>
__global__ void __launch_bounds__(256) memory_output_kernel(const float* __restrict__ o, const T* __restrict__ proj,
                                                            long long ld, int g_off, const float* __restrict__ gain,
                                                            T* __restrict__ y, long long y_ld, int rows, int heads, int vdim,
                                                            int vdim_true, float eps, float out_scale) {
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = static_cast<long long>(blockIdx.x) * 8 + warp;
  if (item >= static_cast<long long>(rows) * heads) return;
  const long long row = item / heads;
  const int head = static_cast<int>(item - row * heads);
  const float* src = o + item * vdim;
  float ss = 0.f;
  for (int c = lane * 4; c < vdim; c += 128) {
    const float4 v = *reinterpret_cast<const float4*>(src + c);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
#pragma unroll
  for (int s = 16; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffff, ss, s);
  const float r = out_scale / sqrtf(ss / vdim_true + eps);
  for (int c = lane * 4; c < vdim; c += 128) {
    const float4 v = *reinterpret_cast<const float4*>(src + c);
    const float4 g = mm_ld4(proj + row * ld + g_off + static_cast<long long>(head) * vdim + c);
    const float4 w = gain ? *reinterpret_cast<const float4*>(gain + head * vdim + c) : g;
    mm_st4(y + row * y_ld + static_cast<long long>(head) * vdim + c, v.x * r * w.x / (1.f + expf(-g.x)),
           v.y * r * w.y / (1.f + expf(-g.y)), v.z * r * w.z / (1.f + expf(-g.z)), v.w * r * w.w / (1.f + expf(-g.w)));
  }
}

// y = o / rms(o over all heads) * gain * sigmoid(g) * out_scale.  One CTA per row; cols = heads * vdim, of which cols_true are in
// use (the others are zero).
template <typename T>
__global__ void __launch_bounds__(256) memory_output_joint_kernel(const float* __restrict__ o, const T* __restrict__ proj,
                                                                  long long ld, int g_off, const float* __restrict__ gain,
                                                                  T* __restrict__ y, long long y_ld, int cols, int cols_true,
                                                                  float eps, float out_scale) {
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  const float* src = o + row * cols;
  constexpr int KEEP = 4;              // groups a thread holds between the two passes; the rest are read again
  float4 v[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = (threadIdx.x + k * 256) * 4;
    v[k] = c < cols ? ld4(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += sq4(v[k]);
  }
  for (int c = (threadIdx.x + KEEP * 256) * 4; c < cols; c += 1024) ss += sq4(ld4(src + c));
  const float r = out_scale / sqrtf(block_sum2(ss, 0.f, red).x / cols_true + eps);
  auto put = [&](int c, const float4& a) {
    const float4 g = mm_ld4(proj + row * ld + g_off + c), w = ld4(gain + c);
    mm_st4(y + row * y_ld + c, a.x * r * w.x / (1.f + expf(-g.x)), a.y * r * w.y / (1.f + expf(-g.y)),
           a.z * r * w.z / (1.f + expf(-g.z)), a.w * r * w.w / (1.f + expf(-g.w)));
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = (threadIdx.x + k * 256) * 4;
    if (c < cols) put(c, v[k]);
  }
  for (int c = (threadIdx.x + KEEP * 256) * 4; c < cols; c += 1024) put(c, ld4(src + c));
}

template <typename T, int R, bool RET>
int launch_scan_r(const ScanParams<T>& p, int segments, cudaStream_t st) {
  const dim3 grid(p.heads * p.slices, segments);
  if (!p.y) {
    launch_k(matrix_memory_scan_kernel<T, R, false, RET>, grid, dim3(MM_THREADS), 0, st, p);
    return launch_status();
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(MM_THREADS);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = p.slices;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = pdl_flag() ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  if (cudaLaunchKernelEx(&cfg, matrix_memory_scan_kernel<T, R, true, RET>, p) != cudaSuccess) {
    const int rc = launch_status();
    return rc ? rc : -7;
  }
  return launch_status();
}

template <typename T, bool RET>
int launch_scan(const ScanParams<T>& p, int segments, cudaStream_t st) {
  if (p.dim <= 32) return launch_scan_r<T, 2, RET>(p, segments, st);
  if (p.dim <= 64) return launch_scan_r<T, 4, RET>(p, segments, st);
  if (p.dim <= 128) return launch_scan_r<T, 8, RET>(p, segments, st);
  if (p.dim <= 256) return launch_scan_r<T, 16, RET>(p, segments, st);
  if (p.dim <= 512) return launch_scan_r<T, 32, RET>(p, segments, st);
  return -2;
}

}  // namespace gk

using namespace gk;

// ptrs: {proj, h, gate_w, gates, gate_b, cu, first_pos, slots, S, n, m, out, y, gain, decay, turns}; y (finished output, one
// row per segment, at most 512 value columns, rows y_ld apart) replaces out; decay (retention) replaces h to gate_b, n, m, gain;
// turns: retention with rot.  dims: {segments, q_off, k_off, v_off, width, heads, dim, vdim, g_off, vdim_true, rot, act}
// floats: {cap, q_scale, eps, out_scale}
GK_EXPORT int gk_matrix_memory_scan(int is_fp32, void* const* ptrs, long long ld, long long y_ld, const int* dims,
                                    const float* floats, void* stream) {
  if (dims[0] == 0) return 0;
  const bool ret = ptrs[14] != nullptr;
  if (dims[7] % 4 || ld % 4 || dims[3] % 4 || (!ret && !ptrs[3] && dims[4] % 4)) return -1;
  if (ptrs[12] && (ptrs[5] || dims[7] > 8 * MM_SLICE || (!ret && !ptrs[13]))) return -3;
  if (!ret && (!ptrs[4] || !ptrs[9] || !ptrs[10])) return -4;
  if (dims[10] < 0 || dims[10] % 2 || dims[10] > dims[6] || dims[10] > MM_MAX_ROT || (dims[10] && !ptrs[15]) ||
      (!ret && (dims[10] || dims[11])) || (dims[10] && dims[11]))
    return -5;
  auto fill = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    ScanParams<T> p;
    p.proj = static_cast<const T*>(ptrs[0]);
    p.ld = ld;
    p.h = static_cast<const T*>(ptrs[1]);
    p.gate_w = static_cast<const T*>(ptrs[2]);
    p.gates = static_cast<const float*>(ptrs[3]);
    p.gate_b = static_cast<const float*>(ptrs[4]);
    p.cu = static_cast<const int*>(ptrs[5]);
    p.first_pos = static_cast<const int*>(ptrs[6]);
    p.slots = static_cast<const int*>(ptrs[7]);
    p.S = static_cast<float*>(ptrs[8]);
    p.n = static_cast<float*>(ptrs[9]);
    p.m = static_cast<float*>(ptrs[10]);
    p.out = static_cast<float*>(ptrs[11]);
    p.y = static_cast<T*>(ptrs[12]);
    p.gain = static_cast<const float*>(ptrs[13]);
    p.decay = static_cast<const float*>(ptrs[14]);
    p.g_off = dims[8]; p.vdim_true = dims[9]; p.eps = floats[2]; p.y_ld = y_ld;
    p.turns = static_cast<const float2*>(ptrs[15]); p.rot = dims[10]; p.act = dims[11];
    p.q_off = dims[1]; p.k_off = dims[2]; p.v_off = dims[3];
    p.width = dims[4]; p.heads = dims[5]; p.dim = dims[6]; p.vdim = dims[7];
    p.slices = (p.vdim + MM_SLICE - 1) / MM_SLICE;
    p.cap = floats[0]; p.q_scale = floats[1]; p.out_scale = floats[3];
    cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
    return ret ? launch_scan<T, true>(p, dims[0], st) : launch_scan<T, false>(p, dims[0], st);
  };
  return is_fp32 ? fill(static_cast<float*>(nullptr)) : fill(static_cast<__nv_bfloat16*>(nullptr));
}

// gain null: no gain, silu in place of the sigmoid.  dims: {rows, heads, vdim, vdim_true, g_off}
GK_EXPORT int gk_memory_output(int is_fp32, const float* o, const void* proj, long long ld, const float* gain, void* y,
                               long long y_ld, const int* dims, float eps, float out_scale, void* stream) {
  const long long items = static_cast<long long>(dims[0]) * dims[1];
  if (items == 0) return 0;
  if (dims[2] % 4 || ld % 4 || y_ld % 4 || dims[4] % 4) return -1;
  const dim3 grid(static_cast<unsigned>((items + 7) / 8));
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (is_fp32)
    launch_k(memory_output_kernel<float>, grid, dim3(256), 0, st, o, static_cast<const float*>(proj), ld, dims[4], gain,
             static_cast<float*>(y), y_ld, dims[0], dims[1], dims[2], dims[3], eps, out_scale);
  else
    launch_k(memory_output_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, o, static_cast<const __nv_bfloat16*>(proj), ld,
             dims[4], gain, static_cast<__nv_bfloat16*>(y), y_ld, dims[0], dims[1], dims[2], dims[3], eps, out_scale);
  return launch_status();
}

// All heads normed together.  dims: {rows, cols, cols_true, g_off};  floats: {eps, out_scale}
GK_EXPORT int gk_memory_output_joint(int is_fp32, const float* o, const void* proj, long long ld, const float* gain, void* y,
                                     long long y_ld, const int* dims, const float* floats, void* stream) {
  if (dims[0] == 0) return 0;
  if (dims[1] < 4 || dims[1] % 4 || dims[2] < 1 || dims[2] > dims[1] || ld % 4 || y_ld % 4 || dims[3] % 4 || !gain) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  auto go = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    launch_k(memory_output_joint_kernel<T>, dim3(dims[0]), dim3(256), 0, st, o, static_cast<const T*>(proj), ld, dims[3], gain,
             static_cast<T*>(y), y_ld, dims[1], dims[2], floats[0], floats[1]);
    return launch_status();
  };
  return is_fp32 ? go(static_cast<float*>(nullptr)) : go(static_cast<__nv_bfloat16*>(nullptr));
}
