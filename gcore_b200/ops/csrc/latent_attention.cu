// Steps around the latent-attention kernels of served decoders (attention_fwd.cu for prompt portions, mla_decode.cu for
// single tokens, window_attention.cu for 32-bit models and other sizes).  A cached row is [latent, normed | key part rotated
// at its position], both padded with zeros; it serves every head.
//   * latent_prep_kernel    a packed projection row -> its cache row (norm of the latent in 32-bit, rotation), the queries'
//                           rotated parts in place, and a copy of the cache row in the portion's contiguous context;
//   * latent_gather_kernel  cache rows of the tokens in front of a portion -> the portion's contiguous context;
//   * gate_columns_kernel   attention output times the sigmoid of a gate per element.
// A portion's context starts at position 0 or, under a window, at the first position its first row sees.  The rotation pairs
// dimension 2i with 2i + 1 (rotary.cuh).
#include "host_utils.h"
#include "rotary.cuh"
#include "row_ops.cuh"
#include <type_traits>

namespace gk {

constexpr int LP_THREADS = 128;
constexpr int LP_MAX_ROT = 256;

__device__ __forceinline__ float lp_f(float v) { return v; }
__device__ __forceinline__ float lp_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void lp_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void lp_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

template <typename T>
struct LatentPrepParams {
  T* proj;                 // packed projection rows
  long long ld;
  int q_off, q_hs;         // head h: unrotated columns at q_off + h * q_hs, rotated ones `q_rot` behind
  int q_rot;
  int d_off;               // latent columns, then the shared key part at d_off + CV
  const float* gain;       // [C]
  const float2* turns;     // [rot / 2] turns per position: value, remainder
  const int* pos;
  const int* slots;        // cache slot of every row; negative: not stored
  T* cache;                // rows of CV + DR
  T* context;              // [context rows, CV + DR] or null
  const int* row_seq;      // with context: portion of every row
  const int* cu_ctx;       //   first context row of every portion
  const int* ctx_start;    //   position of that row, or null: 0
  int rows, context_rows;  //   rows that belong to portions (they come first)
  int H, C, CV, rot, DR;
  float eps, magnitude;
};

// One CTA per row.
template <typename T>
__global__ void __launch_bounds__(LP_THREADS) latent_prep_kernel(const LatentPrepParams<T> p) {
  __shared__ float red[64];
  __shared__ float s_cos[LP_MAX_ROT / 2], s_sin[LP_MAX_ROT / 2];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x, tid = threadIdx.x, half = p.rot >> 1;
  T* pr = p.proj + row * p.ld;
  const int pos = p.pos[row], slot = p.slots[row];
  for (int i = tid; i < half; i += LP_THREADS) {
    float s, c;
    rotation_at(pos, p.turns[i], &s, &c);
    s_cos[i] = c * p.magnitude;
    s_sin[i] = s * p.magnitude;
  }
  float ss = 0.f;
  for (int c = tid; c < p.C; c += LP_THREADS) {
    const float v = lp_f(pr[p.d_off + c]);
    ss += v * v;
  }
  const float r = 1.f / sqrtf(block_sum2(ss, 0.f, red).x / p.C + p.eps);      // also orders the angles for all threads
  const int width = p.CV + p.DR;
  T* dst = slot >= 0 ? p.cache + static_cast<long long>(slot) * width : nullptr;
  T* ctx = nullptr;
  if (p.context && row < p.context_rows) {
    const int b = p.row_seq[row];
    ctx = p.context + (static_cast<long long>(p.cu_ctx[b]) + pos - (p.ctx_start ? p.ctx_start[b] : 0)) * width;
  }
  for (int c = tid; c < width; c += LP_THREADS) {
    float v = 0.f;
    if (c < p.C) {
      v = lp_f(pr[p.d_off + c]) * r * p.gain[c];
    } else if (c >= p.CV && c - p.CV < p.rot) {
      const int i = (c - p.CV) >> 1;
      const float a = lp_f(pr[p.d_off + p.CV + 2 * i]), b = lp_f(pr[p.d_off + p.CV + 2 * i + 1]);
      v = (c - p.CV) & 1 ? b * s_cos[i] + a * s_sin[i] : a * s_cos[i] - b * s_sin[i];
    }
    if (dst) lp_st(dst + c, v);
    if (ctx) lp_st(ctx + c, v);
  }
  for (int i = tid; i < p.H * half; i += LP_THREADS) {
    const int h = i / half, j = i - h * half;
    T* q = pr + p.q_off + static_cast<long long>(h) * p.q_hs + p.q_rot + 2 * j;
    const float a = lp_f(q[0]), b = lp_f(q[1]);
    lp_st(q, a * s_cos[j] - b * s_sin[j]);
    lp_st(q + 1, b * s_cos[j] + a * s_sin[j]);
  }
}

// grid (row groups, portions); one warp per cached row, rows of `vec` 16-byte units
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* __restrict__ cache, const int* __restrict__ tables,
                                                            int max_blocks, int block_size,
                                                            const int* __restrict__ first_pos,
                                                            const int* __restrict__ cu_ctx,
                                                            const int* __restrict__ ctx_start,
                                                            uint4* __restrict__ context, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, start = ctx_start ? ctx_start[b] : 0, n = first_pos[b] - start, lane = threadIdx.x & 31;
  const int* table = tables + static_cast<long long>(b) * max_blocks;
  uint4* out = context + static_cast<long long>(cu_ctx[b]) * vec;
  for (int j = blockIdx.x * 8 + (threadIdx.x >> 5); j < n; j += gridDim.x * 8) {
    const int at = start + j;
    const uint4* src = cache + (static_cast<long long>(table[at / block_size]) * block_size + at % block_size) * vec;
    uint4* dst = out + static_cast<long long>(j) * vec;
    for (int c = lane; c < vec; c += 32) dst[c] = src[c];
  }
}

// x[r, c] *= sigmoid(gate[r, c]), four columns per thread
template <typename T>
__global__ void __launch_bounds__(256) gate_columns_kernel(T* __restrict__ x, long long x_ld, const T* __restrict__ gate,
                                                           long long gate_ld, int rows, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < static_cast<long long>(rows) * vec;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = i / vec;
    const int c = static_cast<int>(i - r * vec) * 4;
    float4 v = ld4(x + r * x_ld + c);
    const float4 g = ld4(gate + r * gate_ld + c);
    v.x /= 1.f + expf(-g.x); v.y /= 1.f + expf(-g.y); v.z /= 1.f + expf(-g.z); v.w /= 1.f + expf(-g.w);
    st4(x + r * x_ld + c, v);
  }
}

}  // namespace gk

using namespace gk;

// ptrs: {proj, gain, turns, pos, slots, cache, context, row_seq, cu_ctx, ctx_start}; context null: single tokens only;
// ctx_start null: contexts start at position 0
// dims: {rows, context_rows, q_off, q_hs, q_rot, d_off, H, C, CV, rot, DR}
GK_EXPORT int gk_latent_prep(int is_fp32, void* const* ptrs, long long ld, const int* dims, float eps, float magnitude,
                             void* stream) {
  if (dims[0] == 0) return 0;
  if (dims[9] % 2 || dims[9] > LP_MAX_ROT || dims[9] > dims[10] || dims[7] > dims[8] || dims[7] < 1) return -1;
  if (ptrs[6] && (!ptrs[7] || !ptrs[8])) return -2;
  auto fill = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    LatentPrepParams<T> p;
    p.proj = static_cast<T*>(ptrs[0]);
    p.ld = ld;
    p.gain = static_cast<const float*>(ptrs[1]);
    p.turns = static_cast<const float2*>(ptrs[2]);
    p.pos = static_cast<const int*>(ptrs[3]);
    p.slots = static_cast<const int*>(ptrs[4]);
    p.cache = static_cast<T*>(ptrs[5]);
    p.context = static_cast<T*>(ptrs[6]);
    p.row_seq = static_cast<const int*>(ptrs[7]);
    p.cu_ctx = static_cast<const int*>(ptrs[8]);
    p.ctx_start = static_cast<const int*>(ptrs[9]);
    p.rows = dims[0]; p.context_rows = dims[1]; p.q_off = dims[2]; p.q_hs = dims[3]; p.q_rot = dims[4]; p.d_off = dims[5];
    p.H = dims[6]; p.C = dims[7]; p.CV = dims[8]; p.rot = dims[9]; p.DR = dims[10];
    p.eps = eps; p.magnitude = magnitude;
    launch_k(latent_prep_kernel<T>, dim3(dims[0]), dim3(LP_THREADS), 0, reinterpret_cast<cudaStream_t>(stream), p);
    return launch_status();
  };
  return is_fp32 ? fill(static_cast<float*>(nullptr)) : fill(static_cast<__nv_bfloat16*>(nullptr));
}

// Rows ctx_start[b] (null: 0) .. first_pos[b] - 1 of every portion's request from the paged cache to its context; max_rows
// bounds their number.
GK_EXPORT int gk_latent_gather(const void* cache, const int* tables, const int* first_pos, const int* cu_ctx,
                               const int* ctx_start, void* context, int portions, int max_blocks, int block_size,
                               int row_bytes, int max_rows, void* stream) {
  if (row_bytes % 16) return -1;
  if (portions == 0 || max_rows == 0) return 0;
  int blocks = (max_rows + 7) / 8;
  if (blocks > sm_count() * 4) blocks = sm_count() * 4;
  launch_k(latent_gather_kernel, dim3(blocks, portions), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream),
           static_cast<const uint4*>(cache), tables, max_blocks, block_size, first_pos, cu_ctx, ctx_start,
           static_cast<uint4*>(context), row_bytes / 16);
  return launch_status();
}

// Columns, strides: multiples of 4 elements, rows 8- (bf16) or 16-byte (32-bit) aligned.
GK_EXPORT int gk_gate_columns(int is_fp32, void* x, long long x_ld, const void* gate, long long gate_ld, int rows, int cols,
                              void* stream) {
  if (cols % 4 || x_ld % 4 || gate_ld % 4) return -1;
  if (rows == 0 || cols == 0) return 0;
  long long blocks = (static_cast<long long>(rows) * (cols / 4) + 255) / 256;
  if (blocks > sm_count() * 8) blocks = sm_count() * 8;
  const dim3 grid(static_cast<unsigned>(blocks)), block(256);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (is_fp32)
    launch_k(gate_columns_kernel<float>, grid, block, 0, st, static_cast<float*>(x), x_ld, static_cast<const float*>(gate),
             gate_ld, rows, cols / 4);
  else
    launch_k(gate_columns_kernel<__nv_bfloat16>, grid, block, 0, st, static_cast<__nv_bfloat16*>(x), x_ld,
             static_cast<const __nv_bfloat16*>(gate), gate_ld, rows, cols / 4);
  return launch_status();
}
