// Residual steps of pre-norm decoders whose sublayers read a short causal convolution over time of their normed input.  One
// launch takes a sublayer's output y to the next sublayer's input:
//     x_t <- x_t + mult * y_t;   n_t = norm(x_t) * gain;   h_t <- sum_j w[j] n_(t - TAPS + 1 + j)
// x, the norm and the convolution are 32-bit.  A request keeps its last TAPS - 1 rows n in 32-bit, position p in ring row
// p mod (TAPS - 1); rows ahead of position 0 are zero.
//
// One CTA = a strip of rows of one portion (or one single token); the TAPS - 1 rows in front of a strip are normed once more
// by it, so strips need nothing from one another, which is also why the new residual goes to another buffer.  Strips start at
// the portion's first row and are at least TAPS - 1 rows long: only the first one reads the ring, and it also writes it, once
// its own rows are done, norming the portion's last rows itself where they lie in another strip.
#include "host_utils.h"
#include "row_ops.cuh"
#include <type_traits>

namespace gk {

template <typename T>
struct ConvNormParams {
  const long long* tokens;  // with embed: x is the token's embedding
  const T* embed;
  const float* x;           // [rows, H] residual, or null with embed
  const T* y;               // [rows, H] sublayer output, or null
  float* x_out;             // [rows, H] new residual, or null
  const float* gain;        // with h
  const float* taps;        // [TAPS, H], or null: the norm itself
  float* ring;              // [slots, TAPS - 1, H]
  const int* cu;            // [n_portions + 1]
  const int* first_pos;     // per portion and single token
  const int* states;        // ring slot, likewise; negative: none
  const long long* pick;    // without taps: source row of every output row, or null
  T* h;                     // [rows, H] or null
  int rows, H, H_true, n_portions, portion_rows, strips, strip, vocab, center;
  float mult, eps;
};

// Block-wide sum with one barrier.  Calls alternate between two buffers: a thread that writes one has passed the barrier of the
// call between, so every thread has read what the buffer held.
__device__ __forceinline__ float cn_sum(float a, float (*red)[32], int& turn) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffff, a, o);
  float* r = red[turn];
  turn ^= 1;
  if (lane == 0) r[w] = a;
  __syncthreads();
  a = lane < nw ? r[lane] : 0.f;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffff, a, o);
  return a;
}

// Thread i owns the float4 groups i, i + blockDim, ... (NV of them).  TAPS 1: no convolution.
template <typename T, int TAPS, int NV>
__global__ void __launch_bounds__(TAPS > 4 ? 1024 : 512) conv_norm_kernel(const ConvNormParams<T> p) {
  constexpr int W = TAPS - 1;
  __shared__ float red[2][32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, nv = p.H >> 2;
  int lo, hi, r_beg, r_end, p0 = 0, slot = -1;
  bool first = false;
  if (TAPS == 1) {
    lo = r_beg = blockIdx.x * p.strip;
    hi = r_end = lo + p.strip < p.rows ? lo + p.strip : p.rows;
  } else {
    const int b = blockIdx.x, in_portions = p.n_portions * p.strips;
    int seg, s = 0;
    if (b < in_portions) {
      seg = b / p.strips;
      s = b - seg * p.strips;
      r_beg = p.cu[seg];
      r_end = p.cu[seg + 1];
    } else {
      seg = p.n_portions + (b - in_portions);
      r_beg = p.portion_rows + (b - in_portions);
      r_end = r_beg + 1;
    }
    lo = r_beg + s * p.strip;
    if (lo >= r_end) return;
    hi = lo + p.strip < r_end ? lo + p.strip : r_end;
    first = s == 0;
    p0 = p.first_pos[seg];
    slot = p.states[seg];
  }

  float4 gain[NV], taps[TAPS <= 4 ? TAPS : 1][NV], win[W > 0 ? W : 1][NV];
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = tid + v * blockDim.x;
    gain[v] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < nv && p.gain) gain[v] = ld4(p.gain + i * 4);
    if (TAPS > 1 && TAPS <= 4) {
#pragma unroll
      for (int j = 0; j < (TAPS <= 4 ? TAPS : 1); ++j)
        taps[j][v] = i < nv ? ld4(p.taps + static_cast<long long>(j) * p.H + i * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }

  // residual of a row, and (y) what is added to it
  auto load = [&](int r, float4 (&x)[NV], float4 (&y)[NV]) {
    const T* e = nullptr;
    const float* xs = nullptr;
    if (p.embed) {
      long long tok = p.tokens[r];
      tok = tok < 0 ? 0 : (tok >= p.vocab ? p.vocab - 1 : tok);
      e = p.embed + tok * p.H;
    } else {
      xs = p.x + (TAPS == 1 && p.pick ? p.pick[r] : static_cast<long long>(r)) * p.H;
    }
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int i = tid + v * blockDim.x;
      x[v] = y[v] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i >= nv) continue;
      x[v] = e ? ld4(e + i * 4) : ld4(xs + i * 4);
      if (p.y) y[v] = ld4(p.y + static_cast<long long>(r) * p.H + i * 4);
    }
  };
  int turn = 0;
  // n of a row whose residual is loaded; x becomes n
  auto norm = [&](int r, float4 (&x)[NV], const float4 (&y)[NV], bool store) {
    float s = 0.f;
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int i = tid + v * blockDim.x;
      x[v].x = fmaf(p.mult, y[v].x, x[v].x); x[v].y = fmaf(p.mult, y[v].y, x[v].y);
      x[v].z = fmaf(p.mult, y[v].z, x[v].z); x[v].w = fmaf(p.mult, y[v].w, x[v].w);
      if (store && i < nv) st4(p.x_out + static_cast<long long>(r) * p.H + i * 4, x[v]);
      s += (x[v].x + x[v].y) + (x[v].z + x[v].w);      // columns past H_true are zero
    }
    if (!p.h) return;
    if (p.center) {
      const float mean = cn_sum(s, red, turn) / p.H_true;
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int c = (tid + v * blockDim.x) * 4;
        x[v].x = c < p.H_true ? x[v].x - mean : 0.f;
        x[v].y = c + 1 < p.H_true ? x[v].y - mean : 0.f;
        x[v].z = c + 2 < p.H_true ? x[v].z - mean : 0.f;
        x[v].w = c + 3 < p.H_true ? x[v].w - mean : 0.f;
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int v = 0; v < NV; ++v) ss += sq4(x[v]);
    const float f = 1.f / sqrtf(cn_sum(ss, red, turn) / p.H_true + p.eps);
#pragma unroll
    for (int v = 0; v < NV; ++v)
      x[v] = make_float4(x[v].x * f * gain[v].x, x[v].y * f * gain[v].y, x[v].z * f * gain[v].z, x[v].w * f * gain[v].w);
  };
  auto ring_row = [&](int pos) { return p.ring + (static_cast<long long>(slot) * (W > 0 ? W : 1) + pos % (W > 0 ? W : 1)) * p.H; };
  auto store_ring = [&](int pos, const float4 (&n)[NV]) {
    float* dst = ring_row(pos);
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int i = tid + v * blockDim.x;
      if (i < nv) st4(dst + i * 4, n[v]);
    }
  };

  // the rows in front of the strip
#pragma unroll
  for (int k = 0; k < W; ++k) {
    const int r = lo - W + k;
    if (r >= r_beg) {
      float4 y[NV];
      load(r, win[k], y);
      norm(r, win[k], y, false);
    } else {
      const int pos = p0 + (r - r_beg);
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int i = tid + v * blockDim.x;
        win[k][v] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < nv && pos >= 0 && slot >= 0) win[k][v] = ld4(ring_row(pos) + i * 4);
      }
    }
  }

  float4 x[NV], y[NV];
  load(lo, x, y);
  for (int r = lo; r < hi; ++r) {
    float4 xn[NV], yn[NV];
    if (r + 1 < hi) {
      load(r + 1, xn, yn);             // on their way while this row is reduced
    } else {
#pragma unroll
      for (int v = 0; v < NV; ++v) xn[v] = yn[v] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    norm(r, x, y, p.x_out != nullptr);
    if (p.h) {
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int i = tid + v * blockDim.x;
        if (i >= nv) continue;
        float4 o = x[v];
        if (TAPS > 1) {
          o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (int j = 0; j < TAPS; ++j) {
            const float4 w = TAPS <= 4 ? taps[TAPS <= 4 ? j : 0][v] : ld4(p.taps + static_cast<long long>(j) * p.H + i * 4);
            const float4 n = j < W ? win[j < W ? j : 0][v] : x[v];
            o.x = fmaf(w.x, n.x, o.x); o.y = fmaf(w.y, n.y, o.y); o.z = fmaf(w.z, n.z, o.z); o.w = fmaf(w.w, n.w, o.w);
          }
        }
        st4(p.h + static_cast<long long>(r) * p.H + i * 4, o);
      }
    }
#pragma unroll
    for (int v = 0; v < NV; ++v) {
#pragma unroll
      for (int k = 0; k + 1 < W; ++k) win[k][v] = win[k + 1][v];
      if (W > 0) win[W > 0 ? W - 1 : 0][v] = x[v];
      x[v] = xn[v];
      y[v] = yn[v];
    }
  }

  if (TAPS > 1 && first && slot >= 0) {
#pragma unroll
    for (int k = 0; k < W; ++k) {
      const int r = r_end - W + k;
      if (r < r_beg) continue;         // an older row: it is in the ring already
      if (hi < r_end) {
        float4 n[NV], z[NV];
        load(r, n, z);
        norm(r, n, z, false);
        store_ring(p0 + (r - r_beg), n);
      } else {
        store_ring(p0 + (r - r_beg), win[k]);
      }
    }
  }
}

template <typename T, int TAPS>
int launch_cn(ConvNormParams<T>& p, int max_portion, cudaStream_t st) {
  const int groups = p.H / 4;
  int threads, per;
  if (TAPS > 4) {
    threads = groups <= 1024 ? (groups + 31) / 32 * 32 : 1024;
    per = (groups + threads - 1) / threads;
  } else {
    per = groups <= 128 ? 1 : 2;
    threads = ((groups + per - 1) / per + 31) / 32 * 32;
    if (threads > 512) {
      threads = 512;
      per = (groups + threads - 1) / threads;
    }
  }
  // strips that fill the GPU a few times over, long enough that the rows in front of them weigh little
  const int most = TAPS > 4 ? 32 : 16;
  int strip = p.rows / (sm_count() * 4);
  strip = strip < 1 ? 1 : strip > most ? most : strip;
  if (strip < TAPS - 1) strip = TAPS - 1;
  p.strip = strip;
  int blocks;
  if (TAPS == 1) {
    blocks = (p.rows + strip - 1) / strip;
  } else {
    p.strips = (max_portion + strip - 1) / strip;
    blocks = p.n_portions * p.strips + (p.rows - p.portion_rows);
  }
  const dim3 grid(blocks), block(threads);
  if (per <= 1) launch_k(conv_norm_kernel<T, TAPS, 1>, grid, block, 0, st, p);
  else if (per <= 2) launch_k(conv_norm_kernel<T, TAPS, 2>, grid, block, 0, st, p);
  else if (per <= 4 && TAPS <= 4) launch_k(conv_norm_kernel<T, TAPS <= 4 ? TAPS : 1, 4>, grid, block, 0, st, p);
  else return -2;
  return launch_status();
}

}  // namespace gk

using namespace gk;

// ptrs: {tokens, embed, x, y, x_out, gain, taps, ring, cu, first_pos, states, pick, h}
// dims: {rows, H, H_true, n_portions, portion_rows, max_portion, n_taps, vocab, center};  n_taps 0: no convolution, else 2, 3, 4,
// 8 or 16;  H % 4 == 0, H <= 8192.  x_out must not overlap x.  floats: {mult, eps}
GK_EXPORT int gk_conv_norm(int is_fp32, void* const* ptrs, const int* dims, const float* floats, void* stream) {
  const int rows = dims[0], H = dims[1], n_taps = dims[6];
  if (rows == 0) return 0;
  if (rows < 0 || H <= 0 || H % 4 || dims[2] < 1 || dims[2] > H) return -1;
  if (ptrs[1] ? (!ptrs[0] || dims[7] < 1 || ptrs[11]) : !ptrs[2]) return -1;
  if ((ptrs[2] && ptrs[2] == ptrs[4]) || (ptrs[12] && !ptrs[5]) || (!ptrs[12] && !ptrs[4])) return -1;
  if (n_taps && (!ptrs[6] || !ptrs[7] || !ptrs[9] || !ptrs[10] || !ptrs[12] || ptrs[11])) return -1;
  if (dims[3] < 0 || (dims[3] > 0) != (dims[4] > 0) || dims[4] > rows || (dims[3] > 0 && (!ptrs[8] || dims[5] < 1))) return -1;
  auto fill = [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    ConvNormParams<T> p;
    p.tokens = static_cast<const long long*>(ptrs[0]);
    p.embed = static_cast<const T*>(ptrs[1]);
    p.x = static_cast<const float*>(ptrs[2]);
    p.y = static_cast<const T*>(ptrs[3]);
    p.x_out = static_cast<float*>(ptrs[4]);
    p.gain = static_cast<const float*>(ptrs[5]);
    p.taps = static_cast<const float*>(ptrs[6]);
    p.ring = static_cast<float*>(ptrs[7]);
    p.cu = static_cast<const int*>(ptrs[8]);
    p.first_pos = static_cast<const int*>(ptrs[9]);
    p.states = static_cast<const int*>(ptrs[10]);
    p.pick = static_cast<const long long*>(ptrs[11]);
    p.h = static_cast<T*>(ptrs[12]);
    p.rows = rows; p.H = H; p.H_true = dims[2]; p.n_portions = dims[3]; p.portion_rows = dims[4];
    p.strips = 0; p.strip = 1; p.vocab = dims[7]; p.center = dims[8];
    p.mult = floats[0]; p.eps = floats[1];
    cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
    switch (n_taps) {
      case 0: return launch_cn<T, 1>(p, dims[5], st);
      case 2: return launch_cn<T, 2>(p, dims[5], st);
      case 3: return launch_cn<T, 3>(p, dims[5], st);
      case 4: return launch_cn<T, 4>(p, dims[5], st);
      case 8: return launch_cn<T, 8>(p, dims[5], st);
      case 16: return launch_cn<T, 16>(p, dims[5], st);
      default: return -3;
    }
  };
  return is_fp32 ? fill(static_cast<float*>(nullptr)) : fill(static_cast<__nv_bfloat16*>(nullptr));
}
