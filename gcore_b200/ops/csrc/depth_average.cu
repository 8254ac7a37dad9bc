// Residual stream of decoders whose layers add one combined update and hand on a weighted average of everything before:
// with X_0 the embedding output and x the stream in front of layer i,
//     X_(i+1) = x + y [+ sum_k w_k routed_k];    x <- sum_{j <= i+1} a_j X_j;    h <- norm(x)
// in one launch: y is the layer's output projection (mixer and feed-forward summed in the product), the routed rows are
// the outputs of the token's experts, still in expert order.  The stream, every X_j and the average are 32-bit.
#include "host_utils.h"
#include "row_ops.cuh"
#include <type_traits>

namespace gk {

template <typename T>
struct DepthParams {
  const float* x_in;        // [rows, H] stream in front of the layer
  const T* y;               // [rows, H]
  const T* routed;          // [expert rows, H] or null
  const int* dest;          // [rows, K] row of `routed` behind every choice
  const float* weight;      // [rows, K]
  const float* history;     // X_0 .. X_i, `hist_stride` floats apart
  long long hist_stride;
  float* result;            // X_(i+1), or null when no later layer reads it
  const float* avg;         // [n + 1] weights of X_0 .. X_(i+1)
  int n;                    // i + 1: results in the history
  float* x_out;             // [rows, H]
  const float* gain;        // with h: gain of the norm in front of the next layer
  T* h;                     // [rows, H] or null
  int n_rows, H, H_true, K;
  float eps;
};

// One CTA per row; thread i owns the float4 groups i, i + blockDim, ... (NV of them).
template <typename T, int NV>
__global__ void __launch_bounds__(256) depth_average_kernel(const DepthParams<T> p) {
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x, off = row * p.H;
  const int nv = p.H >> 2;
  float4 m[NV], acc[NV];
  const float last = p.avg[p.n];
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = threadIdx.x + v * blockDim.x;
    m[v] = acc[v] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < nv) {
      const float4 a = ld4(p.x_in + off + i * 4), b = ld4(p.y + off + i * 4);
      m[v] = make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w);
    }
  }
  if (p.routed) {
    for (int k = 0; k < p.K; ++k) {
      const float w = p.weight[row * p.K + k];
      const T* src = p.routed + static_cast<long long>(p.dest[row * p.K + k]) * p.H;
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int i = threadIdx.x + v * blockDim.x;
        if (i < nv) {
          const float4 a = ld4(src + i * 4);
          m[v].x = fmaf(w, a.x, m[v].x); m[v].y = fmaf(w, a.y, m[v].y);
          m[v].z = fmaf(w, a.z, m[v].z); m[v].w = fmaf(w, a.w, m[v].w);
        }
      }
    }
  }
#pragma unroll 4
  for (int j = 0; j < p.n; ++j) {
    const float w = p.avg[j];
    const float* src = p.history + j * p.hist_stride + off;
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int i = threadIdx.x + v * blockDim.x;
      if (i < nv) {
        const float4 a = ld4(src + i * 4);
        acc[v].x = fmaf(w, a.x, acc[v].x); acc[v].y = fmaf(w, a.y, acc[v].y);
        acc[v].z = fmaf(w, a.z, acc[v].z); acc[v].w = fmaf(w, a.w, acc[v].w);
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = threadIdx.x + v * blockDim.x;
    if (i < nv) {
      if (p.result) st4(p.result + off + i * 4, m[v]);
      acc[v].x = fmaf(last, m[v].x, acc[v].x); acc[v].y = fmaf(last, m[v].y, acc[v].y);
      acc[v].z = fmaf(last, m[v].z, acc[v].z); acc[v].w = fmaf(last, m[v].w, acc[v].w);
      st4(p.x_out + off + i * 4, acc[v]);
      ss += sq4(acc[v]);
    }
  }
  if (!p.h) return;
  const float r = 1.f / sqrtf(block_sum2(ss, 0.f, red).x / p.H_true + p.eps);
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = threadIdx.x + v * blockDim.x;
    if (i < nv) {
      const float4 g = ld4(p.gain + i * 4);
      st4(p.h + off + i * 4, make_float4(acc[v].x * r * g.x, acc[v].y * r * g.y, acc[v].z * r * g.z, acc[v].w * r * g.w));
    }
  }
}

template <typename T>
int launch_depth(const DepthParams<T>& p, cudaStream_t st) {
  const int threads = p.H <= 512 ? 128 : 256;
  const int per = (p.H / 4 + threads - 1) / threads;
  const dim3 grid(p.n_rows);
  if (per <= 1) launch_k(depth_average_kernel<T, 1>, grid, dim3(threads), 0, st, p);
  else if (per <= 2) launch_k(depth_average_kernel<T, 2>, grid, dim3(threads), 0, st, p);
  else if (per <= 4) launch_k(depth_average_kernel<T, 4>, grid, dim3(threads), 0, st, p);
  else if (per <= 8) launch_k(depth_average_kernel<T, 8>, grid, dim3(threads), 0, st, p);
  else if (per <= 16) launch_k(depth_average_kernel<T, 16>, grid, dim3(threads), 0, st, p);
  else return -2;
  return launch_status();
}

}  // namespace gk

using namespace gk;

// ptrs: {x_in, y, routed, dest, weight, history, result, avg, x_out, gain, h}
// dims: {n_rows, H, H_true, n, K};  hist_stride in floats
GK_EXPORT int gk_depth_average(int is_fp32, void* const* ptrs, long long hist_stride, const int* dims, float eps,
                               void* stream) {
  if (dims[0] == 0) return 0;
  if (dims[1] % 4 || dims[1] <= 0 || dims[2] <= 0 || dims[2] > dims[1] || dims[3] < 1) return -1;
  auto fill = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    DepthParams<T> p;
    p.x_in = static_cast<const float*>(ptrs[0]);
    p.y = static_cast<const T*>(ptrs[1]);
    p.routed = static_cast<const T*>(ptrs[2]);
    p.dest = static_cast<const int*>(ptrs[3]);
    p.weight = static_cast<const float*>(ptrs[4]);
    p.history = static_cast<const float*>(ptrs[5]);
    p.result = static_cast<float*>(ptrs[6]);
    p.avg = static_cast<const float*>(ptrs[7]);
    p.x_out = static_cast<float*>(ptrs[8]);
    p.gain = static_cast<const float*>(ptrs[9]);
    p.h = static_cast<T*>(ptrs[10]);
    p.hist_stride = hist_stride;
    p.n_rows = dims[0]; p.H = dims[1]; p.H_true = dims[2]; p.n = dims[3]; p.K = dims[4];
    p.eps = eps;
    return launch_depth<T>(p, reinterpret_cast<cudaStream_t>(stream));
  };
  return is_fp32 ? fill(static_cast<float*>(nullptr)) : fill(static_cast<__nv_bfloat16*>(nullptr));
}
