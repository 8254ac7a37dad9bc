// Residual-stream kernels of decoders that normalise before and after every sublayer and keep the residual in 32-bit:
// one launch takes a sublayer's output to the next sublayer's input,
//     x <- x + post_norm(y) [+ embedding output] [+ step vector];   h <- pre_norm(x)
// where y is one tensor, or half the sum of two mixers' outputs each normalised with a gain of its own, and the first
// launch of a forward pass builds x from the token table (and the position table of models that have one) instead.  Norm gains are 32-bit; "one-plus"
// gains are stored as (1 + w) by the loader, so every norm here is x / sqrt(mean(x^2) + eps) * gain.
#include "host_utils.h"
#include "row_ops.cuh"
#include <type_traits>

namespace gk {

enum : int { SRC_EMBED = 0, SRC_ONE = 1, SRC_PAIR = 2, SRC_ROWS = 3 };

template <typename T>
struct SandwichParams {
  const long long* tokens;   // SRC_EMBED
  const int* pos;            // SRC_EMBED
  const T* embed;            // [vocab, H]
  const T* pos_table;        // [max positions, H], or null: tokens alone
  int vocab, max_pos;
  const T* ya;               // SRC_ONE / SRC_PAIR: [rows, H]
  const T* yb;               // SRC_PAIR
  const float* gain_a;       // SRC_PAIR: gains of the two outputs
  const float* gain_b;
  const float* gain_post;    // SRC_ONE / SRC_PAIR
  float* x;                  // residual stream [rows, H]
  float* x_first;            // SRC_EMBED: copy of the embedding output, or null
  const float* x_add;        // embedding output to add, or null
  const float* step;         // [H] vector to add, or null
  const long long* rows;     // SRC_ROWS: row of x behind each output row, or null
  const float* gain_pre;     // with h: gain of the norm in front of the next sublayer
  T* h;                      // [rows, H] or null
  int n_rows, H, H_true;
  float eps;
};

// One CTA per row; thread i owns the float4 groups i, i + blockDim, ... (NV of them).
template <typename T, int SRC, int NV>
__global__ void __launch_bounds__(256) sandwich_norm_kernel(const SandwichParams<T> p) {
  __shared__ float red[64];
  pdl_launch_dependents();
  pdl_wait();
  const long long row = blockIdx.x;
  const long long off = row * p.H;
  const int nv = p.H >> 2;
  const float inv_n = 1.f / p.H_true;
  float4 m[NV];
  long long xoff = off;
  if (SRC == SRC_EMBED) {
    long long tok = p.tokens[row];
    int ps = p.pos_table ? p.pos[row] : 0;
    tok = tok < 0 ? 0 : (tok >= p.vocab ? p.vocab - 1 : tok);      // ids are checked on the host
    ps = ps < 0 ? 0 : (ps >= p.max_pos ? p.max_pos - 1 : ps);
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int i = threadIdx.x + v * blockDim.x;
      m[v] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < nv) {
        m[v] = ld4(p.embed + tok * p.H + i * 4);
        if (p.pos_table) {
          const float4 b = ld4(p.pos_table + static_cast<long long>(ps) * p.H + i * 4);
          m[v].x += b.x; m[v].y += b.y; m[v].z += b.z; m[v].w += b.w;
        }
        if (p.x_first) st4(p.x_first + off + i * 4, m[v]);
      }
    }
  } else if (SRC == SRC_ROWS) {
    if (p.rows) xoff = p.rows[row] * p.H;
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int i = threadIdx.x + v * blockDim.x;
      m[v] = i < nv ? ld4(p.x + xoff + i * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  } else {
    float4 xr[NV];   // the residual is requested together with the sublayer's output
    float sa = 0.f, sb = 0.f;
    float4 u[SRC == SRC_PAIR ? NV : 1];
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int i = threadIdx.x + v * blockDim.x;
      m[v] = xr[v] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (SRC == SRC_PAIR) u[v] = m[v];
      if (i < nv) {
        m[v] = ld4(p.ya + off + i * 4);
        if (SRC == SRC_PAIR) u[v] = ld4(p.yb + off + i * 4);
        xr[v] = ld4(p.x + off + i * 4);
        sa += sq4(m[v]);
        if (SRC == SRC_PAIR) sb += sq4(u[v]);
      }
    }
    float2 s = block_sum2(sa, sb, red);
    if (SRC == SRC_PAIR) {
      const float ra = 0.5f / sqrtf(s.x * inv_n + p.eps), rb = 0.5f / sqrtf(s.y * inv_n + p.eps);
      sa = 0.f;
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int i = threadIdx.x + v * blockDim.x;
        if (i < nv) {
          const float4 ga = ld4(p.gain_a + i * 4), gb = ld4(p.gain_b + i * 4);
          m[v].x = m[v].x * ra * ga.x + u[v].x * rb * gb.x;
          m[v].y = m[v].y * ra * ga.y + u[v].y * rb * gb.y;
          m[v].z = m[v].z * ra * ga.z + u[v].z * rb * gb.z;
          m[v].w = m[v].w * ra * ga.w + u[v].w * rb * gb.w;
          sa += sq4(m[v]);
        }
      }
      s = block_sum2(sa, 0.f, red);
    }
    const float r = 1.f / sqrtf(s.x * inv_n + p.eps);
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int i = threadIdx.x + v * blockDim.x;
      if (i < nv) {
        const float4 g = ld4(p.gain_post + i * 4);
        m[v].x = xr[v].x + m[v].x * r * g.x;
        m[v].y = xr[v].y + m[v].y * r * g.y;
        m[v].z = xr[v].z + m[v].z * r * g.z;
        m[v].w = xr[v].w + m[v].w * r * g.w;
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = threadIdx.x + v * blockDim.x;
    if (i < nv) {
      if (p.x_add) {
        const float4 a = ld4(p.x_add + off + i * 4);
        m[v].x += a.x; m[v].y += a.y; m[v].z += a.z; m[v].w += a.w;
      }
      if (p.step) {
        const float4 a = ld4(p.step + i * 4);
        m[v].x += a.x; m[v].y += a.y; m[v].z += a.z; m[v].w += a.w;
      }
      if (SRC != SRC_ROWS) st4(p.x + off + i * 4, m[v]);
      ss += sq4(m[v]);
    }
  }
  if (!p.h) return;
  const float2 s = block_sum2(ss, 0.f, red);
  const float r = 1.f / sqrtf(s.x * inv_n + p.eps);
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = threadIdx.x + v * blockDim.x;
    if (i < nv) {
      const float4 g = ld4(p.gain_pre + i * 4);
      st4(p.h + off + i * 4, make_float4(m[v].x * r * g.x, m[v].y * r * g.y, m[v].z * r * g.z, m[v].w * r * g.w));
    }
  }
}

template <typename T, int SRC>
int launch_sandwich(const SandwichParams<T>& p, cudaStream_t st) {
  if (p.n_rows == 0) return 0;
  if (p.H % 4 || p.H <= 0 || p.H_true <= 0 || p.H_true > p.H) return -1;
  const dim3 grid(p.n_rows);
  const int threads = p.H <= 512 ? 128 : 256;
  const int per = (p.H / 4 + threads - 1) / threads;
  if (per <= 1) launch_k(sandwich_norm_kernel<T, SRC, 1>, grid, dim3(threads), 0, st, p);
  else if (per <= 2) launch_k(sandwich_norm_kernel<T, SRC, 2>, grid, dim3(threads), 0, st, p);
  else if (per <= 4) launch_k(sandwich_norm_kernel<T, SRC, 4>, grid, dim3(threads), 0, st, p);
  else if (per <= 8) launch_k(sandwich_norm_kernel<T, SRC, 8>, grid, dim3(threads), 0, st, p);
  else if (per <= 16) launch_k(sandwich_norm_kernel<T, SRC, 16>, grid, dim3(threads), 0, st, p);
  else return -2;
  return launch_status();
}

template <typename T>
int sandwich(int src, const SandwichParams<T>& p, cudaStream_t st) {
  switch (src) {
    case SRC_EMBED: return launch_sandwich<T, SRC_EMBED>(p, st);
    case SRC_ONE: return launch_sandwich<T, SRC_ONE>(p, st);
    case SRC_PAIR: return launch_sandwich<T, SRC_PAIR>(p, st);
    case SRC_ROWS: return launch_sandwich<T, SRC_ROWS>(p, st);
  }
  return -3;
}

// silu(gate) * up in 32-bit, for models that run in 32-bit ([gate | up] rows of 2F).
__global__ void swiglu_f32_kernel(const float* __restrict__ in, float* __restrict__ out, long long n, int F) {
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const long long t = i / F, c = i - t * F;
  const float g = in[t * 2 * F + c], u = in[t * 2 * F + F + c];
  out[i] = g / (1.f + expf(-g)) * u;
}

}  // namespace gk

using namespace gk;

// ptrs: {tokens, pos, embed, pos_table, ya, yb, gain_a, gain_b, gain_post, x, x_first, x_add, step, rows, gain_pre, h}
// dims: {vocab, max_pos, n_rows, H, H_true}
GK_EXPORT int gk_sandwich_norm(int src, int is_fp32, void* const* ptrs, const int* dims, float eps, void* stream) {
  auto fill = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    SandwichParams<T> p;
    p.tokens = static_cast<const long long*>(ptrs[0]);
    p.pos = static_cast<const int*>(ptrs[1]);
    p.embed = static_cast<const T*>(ptrs[2]);
    p.pos_table = static_cast<const T*>(ptrs[3]);
    p.ya = static_cast<const T*>(ptrs[4]);
    p.yb = static_cast<const T*>(ptrs[5]);
    p.gain_a = static_cast<const float*>(ptrs[6]);
    p.gain_b = static_cast<const float*>(ptrs[7]);
    p.gain_post = static_cast<const float*>(ptrs[8]);
    p.x = static_cast<float*>(ptrs[9]);
    p.x_first = static_cast<float*>(ptrs[10]);
    p.x_add = static_cast<const float*>(ptrs[11]);
    p.step = static_cast<const float*>(ptrs[12]);
    p.rows = static_cast<const long long*>(ptrs[13]);
    p.gain_pre = static_cast<const float*>(ptrs[14]);
    p.h = static_cast<T*>(ptrs[15]);
    p.vocab = dims[0]; p.max_pos = dims[1]; p.n_rows = dims[2]; p.H = dims[3]; p.H_true = dims[4];
    p.eps = eps;
    return sandwich<T>(src, p, reinterpret_cast<cudaStream_t>(stream));
  };
  return is_fp32 ? fill(static_cast<float*>(nullptr)) : fill(static_cast<__nv_bfloat16*>(nullptr));
}

GK_EXPORT int gk_swiglu_f32(const float* in, float* out, long long T, int F, void* stream) {
  const long long n = T * F;
  if (n == 0) return 0;
  swiglu_f32_kernel<<<static_cast<unsigned>((n + 255) / 256), 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(in, out, n, F);
  return launch_status();
}
