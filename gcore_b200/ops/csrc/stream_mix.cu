// Residual streams of decoders with hyper-connections: S copies x_1 .. x_S of the residual, of which a sublayer reads one
// weighted sum and to all of which it writes.  Between two sublayers, in one launch:
//     x_t <- sum_s mix[s, t] x_s + write[t] * (y [+ sum_k w_k routed_k]);   u = sum_t read[t] x_t;   h <- norm(u) * gain
// y is the sublayer's output projection, the routed rows are the outputs of the token's experts, still in expert order.
// Everything is 32-bit up to the rounding of h.  A row of the streams is [S, H].
#include "host_utils.h"
#include "row_ops.cuh"
#include <type_traits>

namespace gk {

template <typename T>
struct StreamParams {
  float* x;                 // [rows, S, H]
  const long long* tokens;  // with embed: all streams start as the token's embedding
  const T* embed;
  const T* y;               // [rows, H] or null
  const T* routed;          // [expert rows, H] or null
  const int* dest;          // [rows, K] row of `routed` behind every choice
  const float* weight;      // [rows, K]
  const float* mix;         // [S, S], from x to
  const float* write;       // [S]
  const float* read;        // [S], or null: all ones
  const float* gain;        // with h
  T* h;                     // [rows, H] or null
  float* total;             // [rows, H] or null: u itself
  int rows, S, H, H_true, K, vocab, keep;
  float eps;
};

// One CTA per row; thread i owns the float4 groups i, i + blockDim, ... (NV of them) of every stream.  SM: streams the
// registers hold; EXACT: S == SM.
template <typename T, int SM, bool EXACT, int NV>
__global__ void __launch_bounds__(256) stream_mix_kernel(const StreamParams<T> p) {
  __shared__ float red[64];
  __shared__ float s_mix[SM * SM], s_write[SM], s_read[SM];
  const int S = EXACT ? SM : p.S, tid = threadIdx.x;
  // the connections are weights: no earlier kernel of the step writes them
  if (!p.embed) {
    for (int i = tid; i < S * S; i += blockDim.x) s_mix[(i / S) * SM + i % S] = p.mix[i];
    if (tid < S) s_write[tid] = p.write[tid];
  }
  if (tid < S) s_read[tid] = p.read ? p.read[tid] : 1.f;
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();
  const long long row = blockIdx.x;
  const int nv = p.H >> 2;
  float* x = p.x + row * S * p.H;
  const T* src = nullptr;
  if (p.embed) {
    long long tok = p.tokens[row];
    tok = tok < 0 ? 0 : (tok >= p.vocab ? p.vocab - 1 : tok);
    src = p.embed + tok * p.H;
  }
  float4 u[NV];
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = tid + v * blockDim.x;
    u[v] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= nv) continue;
    if (p.embed) {
      const float4 e = ld4(src + i * 4);
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (!EXACT && t >= S) break;
        st4(x + t * p.H + i * 4, e);
        const float r = s_read[t];
        u[v].x = fmaf(r, e.x, u[v].x); u[v].y = fmaf(r, e.y, u[v].y);
        u[v].z = fmaf(r, e.z, u[v].z); u[v].w = fmaf(r, e.w, u[v].w);
      }
    } else {
      float4 old[SM];
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (EXACT || s < S) old[s] = ld4(x + s * p.H + i * 4);
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
      if (p.y) y = ld4(p.y + row * p.H + i * 4);
      for (int k = 0; k < p.K; ++k) {
        const float w = p.weight[row * p.K + k];
        const float4 a = ld4(p.routed + static_cast<long long>(p.dest[row * p.K + k]) * p.H + i * 4);
        y.x = fmaf(w, a.x, y.x); y.y = fmaf(w, a.y, y.y); y.z = fmaf(w, a.z, y.z); y.w = fmaf(w, a.w, y.w);
      }
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (!EXACT && t >= S) break;
        const float o = s_write[t], r = s_read[t];
        float4 n = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
        for (int s = 0; s < SM; ++s) {
          if (!EXACT && s >= S) break;
          const float m = s_mix[s * SM + t];
          n.x = fmaf(m, old[s].x, n.x); n.y = fmaf(m, old[s].y, n.y);
          n.z = fmaf(m, old[s].z, n.z); n.w = fmaf(m, old[s].w, n.w);
        }
        if (p.keep) st4(x + t * p.H + i * 4, n);
        u[v].x = fmaf(r, n.x, u[v].x); u[v].y = fmaf(r, n.y, u[v].y);
        u[v].z = fmaf(r, n.z, u[v].z); u[v].w = fmaf(r, n.w, u[v].w);
      }
    }
    if (p.total) st4(p.total + row * p.H + i * 4, u[v]);
    ss += sq4(u[v]);
  }
  if (!p.h) return;
  const float r = 1.f / sqrtf(block_sum2(ss, 0.f, red).x / p.H_true + p.eps);
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = tid + v * blockDim.x;
    if (i < nv) {
      const float4 g = ld4(p.gain + i * 4);
      st4(p.h + row * p.H + i * 4, make_float4(u[v].x * r * g.x, u[v].y * r * g.y, u[v].z * r * g.z, u[v].w * r * g.w));
    }
  }
}

template <typename T, int SM, bool EXACT>
int launch_streams(const StreamParams<T>& p, cudaStream_t st) {
  const int threads = p.H <= 512 ? 128 : 256;
  const int per = (p.H / 4 + threads - 1) / threads;
  const dim3 grid(p.rows), block(threads);
  if (per <= 1) launch_k(stream_mix_kernel<T, SM, EXACT, 1>, grid, block, 0, st, p);
  else if (per <= 2) launch_k(stream_mix_kernel<T, SM, EXACT, 2>, grid, block, 0, st, p);
  else if (per <= 4) launch_k(stream_mix_kernel<T, SM, EXACT, 4>, grid, block, 0, st, p);
  else if (per <= 16) launch_k(stream_mix_kernel<T, SM, EXACT, 16>, grid, block, 0, st, p);
  else return -2;
  return launch_status();
}

}  // namespace gk

using namespace gk;

// ptrs: {x, tokens, embed, y, routed, dest, weight, mix, write, read, gain, h, total}
// dims: {rows, S, H, H_true, K, vocab, keep};  H % 4 == 0, S <= 16
GK_EXPORT int gk_stream_mix(int is_fp32, void* const* ptrs, const int* dims, float eps, void* stream) {
  if (dims[0] == 0) return 0;
  if (dims[1] < 1 || dims[1] > 16 || dims[2] % 4 || dims[2] <= 0 || dims[3] <= 0 || dims[3] > dims[2]) return -1;
  if (ptrs[2] ? (!ptrs[1] || dims[5] < 1) : (!ptrs[7] || !ptrs[8])) return -1;
  if ((dims[4] > 0) != (ptrs[4] != nullptr) || (ptrs[11] && !ptrs[10])) return -1;
  auto fill = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    StreamParams<T> p;
    p.x = static_cast<float*>(ptrs[0]);
    p.tokens = static_cast<const long long*>(ptrs[1]);
    p.embed = static_cast<const T*>(ptrs[2]);
    p.y = static_cast<const T*>(ptrs[3]);
    p.routed = static_cast<const T*>(ptrs[4]);
    p.dest = static_cast<const int*>(ptrs[5]);
    p.weight = static_cast<const float*>(ptrs[6]);
    p.mix = static_cast<const float*>(ptrs[7]);
    p.write = static_cast<const float*>(ptrs[8]);
    p.read = static_cast<const float*>(ptrs[9]);
    p.gain = static_cast<const float*>(ptrs[10]);
    p.h = static_cast<T*>(ptrs[11]);
    p.total = static_cast<float*>(ptrs[12]);
    p.rows = dims[0]; p.S = dims[1]; p.H = dims[2]; p.H_true = dims[3]; p.K = dims[4]; p.vocab = dims[5]; p.keep = dims[6];
    p.eps = eps;
    cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
    switch (p.S) {
      case 1: return launch_streams<T, 1, true>(p, st);
      case 2: return launch_streams<T, 2, true>(p, st);
      case 3: return launch_streams<T, 3, true>(p, st);
      case 4: return launch_streams<T, 4, true>(p, st);
      default: return p.S <= 8 ? launch_streams<T, 8, false>(p, st) : launch_streams<T, 16, false>(p, st);
    }
  };
  return is_fp32 ? fill(static_cast<float*>(nullptr)) : fill(static_cast<__nv_bfloat16*>(nullptr));
}
