// Feed-forward steps of served layer-plan decoders: activations on packed projections, and what a mixture of experts needs
// around the grouped GEMMs when routing has counted the tokens of every expert (router.cu):
//   * ffn_act_kernel        silu(gate) * up or relu(up)^2, optionally scaled by a sigmoid per row, between two strided
//                           matrices;
//   * expert_rows_kernel    segment offsets (128-row segments, as the grouped GEMM wants them) and the copy of every
//                           token's row into its experts' segments, one launch;
//   * grouped_f32_kernel    the grouped product in true 32-bit, for models that run in 32-bit.
#include "host_utils.h"
#include "row_ops.cuh"
#include <type_traits>

namespace gk {

enum : int { ACT_SILU_GATE = 0, ACT_RELU2 = 1 };

template <typename T>
struct ActParams {
  const T* src;             // gate columns first (ACT_SILU_GATE), `up` columns at up_off
  long long src_ld;
  int up_off;
  T* dst;
  long long dst_ld;
  const float* row_logit;   // one logit per row, `logit_ld` apart: the row is scaled by its sigmoid; or null
  long long logit_ld;
  const int* n_rows_dev;    // rows in use (on the device), or null: all
  long long rows;
  int F;                    // columns, a multiple of 4
};

// 32-bit rows take the exact exponential and quotient, bf16 rows the fast ones (their error is far below the rounding).
__device__ __forceinline__ float act_sigmoid(float z, float) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float act_sigmoid(float z, __nv_bfloat16) { return __fdividef(1.f, 1.f + __expf(-z)); }

template <typename T, int ACT>
__device__ __forceinline__ float4 act4(const T* gate, const T* up, float w) {
  float4 u = ld4(up);
  if (ACT == ACT_SILU_GATE) {
    const float4 g = ld4(gate);
    u.x *= g.x * act_sigmoid(g.x, T()); u.y *= g.y * act_sigmoid(g.y, T());
    u.z *= g.z * act_sigmoid(g.z, T()); u.w *= g.w * act_sigmoid(g.w, T());
  } else {
    u.x = fmaxf(u.x, 0.f); u.y = fmaxf(u.y, 0.f); u.z = fmaxf(u.z, 0.f); u.w = fmaxf(u.w, 0.f);
    u.x *= u.x; u.y *= u.y; u.z *= u.z; u.w *= u.w;
  }
  u.x *= w; u.y *= w; u.z *= w; u.w *= w;
  return u;
}

// grid (column groups of 4 * blockDim.x, row groups): a thread keeps its columns and walks rows, four at a time so that
// their loads overlap.
template <typename T, int ACT>
__global__ void __launch_bounds__(256) ffn_act_kernel(const ActParams<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (c >= p.F) return;
  long long rows = p.rows;
  if (p.n_rows_dev && *p.n_rows_dev < rows) rows = *p.n_rows_dev;
  for (long long r0 = static_cast<long long>(blockIdx.y) * 4; r0 < rows; r0 += static_cast<long long>(gridDim.y) * 4) {
    float4 u[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const long long row = r0 + i < rows ? r0 + i : rows - 1;
      const float w = p.row_logit ? 1.f / (1.f + expf(-p.row_logit[row * p.logit_ld])) : 1.f;
      const T* s = p.src + row * p.src_ld + c;
      u[i] = act4<T, ACT>(s, s + p.up_off, w);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (r0 + i < rows) st4(p.dst + (r0 + i) * p.dst_ld + c, u[i]);
  }
}

constexpr int ER_MAX_EXPERTS = 512;
constexpr int ER_THREADS = 256;

// Every CTA derives all segment offsets from the counts (a few hundred numbers) and copies its share of the rows; one warp
// per (token, choice).  Rows are `row_vec` 16-byte units.
__global__ void __launch_bounds__(ER_THREADS) expert_rows_kernel(const uint4* __restrict__ h, const int* __restrict__ counts,
                                                                 const long long* __restrict__ choice,
                                                                 const int* __restrict__ place, int* __restrict__ offsets,
                                                                 int* __restrict__ dest, uint4* __restrict__ out,
                                                                 int n, int K, int E, int row_vec) {
  __shared__ int s_off[ER_MAX_EXPERTS + 1];
  __shared__ int s_warp[ER_THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  // exclusive prefix sums of the padded counts: two experts per thread
  const int e0 = 2 * tid;
  const int a = e0 < E ? (counts[e0] + 127) / 128 * 128 : 0, b = e0 + 1 < E ? (counts[e0 + 1] + 127) / 128 * 128 : 0;
  int incl = a + b;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int y = __shfl_up_sync(0xffffffff, incl, o);
    if (lane >= o) incl += y;
  }
  if (lane == 31) s_warp[warp] = incl;
  __syncthreads();
  int before = incl - a - b;
  for (int w = 0; w < warp; ++w) before += s_warp[w];
  if (e0 <= E) s_off[e0] = before;
  if (e0 + 1 <= E) s_off[e0 + 1] = before + a;
  if (tid == ER_THREADS - 1 && E == ER_MAX_EXPERTS) s_off[E] = before + a + b;
  __syncthreads();
  if (blockIdx.x == 0)
    for (int e = tid; e <= E; e += ER_THREADS) offsets[e] = s_off[e];
  for (int i = blockIdx.x * (ER_THREADS / 32) + warp; i < n; i += gridDim.x * (ER_THREADS / 32)) {
    const int r = s_off[static_cast<int>(choice[i])] + place[i];
    if (lane == 0) dest[i] = r;
    const uint4* src = h + static_cast<long long>(i / K) * row_vec;
    uint4* dst = out + static_cast<long long>(r) * row_vec;
    for (int c = lane; c < row_vec; c += 32) dst[c] = src[c];
  }
}

// C[r, :] = A[r, :] W[g]^T for the rows r of segment g.  64 x 64 tiles, 4 x 4 outputs per thread; A [rows, K],
// W [G, N, K], both row-major 32-bit.
constexpr int GF_T = 64, GF_K = 16;
__global__ void __launch_bounds__(256) grouped_f32_kernel(const float* __restrict__ A, const float* __restrict__ W,
                                                          float* __restrict__ C, const int* __restrict__ offsets, int G,
                                                          int N, int K) {
  __shared__ float sa[GF_K][GF_T + 4], sw[GF_K][GF_T + 4];
  const int m0 = blockIdx.y * GF_T, n0 = blockIdx.x * GF_T;
  if (m0 >= offsets[G]) return;
  int g = 0;
  while (g + 1 < G && offsets[g + 1] <= m0) ++g;      // segments are multiples of 128 rows: a tile lies in one
  const float* w = W + static_cast<long long>(g) * N * K;
  const int tid = threadIdx.x, tr = (tid >> 4) * 4, tc = (tid & 15) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += GF_K) {
    for (int i = tid; i < GF_T * GF_K; i += 256) {
      const int r = i / GF_K, k = i % GF_K;
      sa[k][r] = k0 + k < K ? A[static_cast<long long>(m0 + r) * K + k0 + k] : 0.f;
      sw[k][r] = k0 + k < K && n0 + r < N ? w[static_cast<long long>(n0 + r) * K + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GF_K; ++k) {
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(sa[k][tr + x], sw[k][tc + y], acc[x][y]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int x = 0; x < 4; ++x)
#pragma unroll
    for (int y = 0; y < 4; ++y)
      if (n0 + tc + y < N) C[static_cast<long long>(m0 + tr + x) * N + n0 + tc + y] = acc[x][y];
}

template <typename T>
int launch_act(int act, const ActParams<T>& p, cudaStream_t st) {
  const int cols = p.F >> 2;
  const int threads = cols >= 256 ? 256 : (cols + 31) / 32 * 32;
  const unsigned gx = static_cast<unsigned>((cols + threads - 1) / threads);
  long long gy = (p.rows + 3) / 4;
  const long long most = (sm_count() * 16 + gx - 1) / gx;
  if (gy > most) gy = most;
  const dim3 grid(gx, static_cast<unsigned>(gy)), block(threads);
  if (act == ACT_SILU_GATE) launch_k(ffn_act_kernel<T, ACT_SILU_GATE>, grid, block, 0, st, p);
  else if (act == ACT_RELU2) launch_k(ffn_act_kernel<T, ACT_RELU2>, grid, block, 0, st, p);
  else return -3;
  return launch_status();
}

}  // namespace gk

using namespace gk;

// ptrs: {src, dst, row_logit, n_rows_dev};  lds: {src_ld, dst_ld, logit_ld, rows};  dims: {up_off, F}
GK_EXPORT int gk_ffn_act(int act, int is_fp32, void* const* ptrs, const long long* lds, const int* dims, void* stream) {
  if (lds[3] == 0) return 0;
  if (dims[0] % 4 || dims[1] % 4 || lds[0] % 4 || lds[1] % 4) return -1;
  auto fill = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    ActParams<T> p;
    p.src = static_cast<const T*>(ptrs[0]);
    p.dst = static_cast<T*>(ptrs[1]);
    p.row_logit = static_cast<const float*>(ptrs[2]);
    p.n_rows_dev = static_cast<const int*>(ptrs[3]);
    p.src_ld = lds[0]; p.dst_ld = lds[1]; p.logit_ld = lds[2]; p.rows = lds[3];
    p.up_off = dims[0]; p.F = dims[1];
    return launch_act<T>(act, p, reinterpret_cast<cudaStream_t>(stream));
  };
  return is_fp32 ? fill(static_cast<float*>(nullptr)) : fill(static_cast<__nv_bfloat16*>(nullptr));
}

// choice, place: [tokens * K]; out: room for every token's rows with the segments padded to 128.  row_bytes % 16 == 0.
GK_EXPORT int gk_expert_rows(const void* h, const int* counts, const long long* choice, const int* place, int* offsets,
                             int* dest, void* out, int tokens, int K, int E, int row_bytes, void* stream) {
  if (E < 1 || E > ER_MAX_EXPERTS || K < 1 || row_bytes % 16) return -1;
  const int n = tokens * K;
  int blocks = (n + ER_THREADS / 32 - 1) / (ER_THREADS / 32);
  if (blocks > sm_count() * 8) blocks = sm_count() * 8;
  if (blocks < 1) blocks = 1;
  launch_k(expert_rows_kernel, dim3(blocks), dim3(ER_THREADS), 0, reinterpret_cast<cudaStream_t>(stream),
           static_cast<const uint4*>(h), counts, choice, place, offsets, dest, static_cast<uint4*>(out), n, K, E,
           row_bytes / 16);
  return launch_status();
}

// rows: rows of A and C (a multiple of 64); offsets [G + 1] on the device, multiples of 128
GK_EXPORT int gk_grouped_gemm_f32(const float* A, const float* W, float* C, const int* offsets, int G, int rows, int N,
                                  int K, void* stream) {
  if (rows % GF_T || N < 1 || K < 1 || rows / GF_T > 65535) return -1;
  if (rows == 0) return 0;
  grouped_f32_kernel<<<dim3((N + GF_T - 1) / GF_T, rows / GF_T), 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(
      A, W, C, offsets, G, N, K);
  return launch_status();
}
