// Residual steps of pre-norm decoders whose sublayers read a short causal convolution over time of their normed input.  One
// launch takes a sublayer's output y to the next sublayer's input:
//     x_t <- x_t + mult * y_t;   n_t = norm(x_t) * gain;   h_t <- sum_j w[j] n_(t - TAPS + 1 + j)
// x, the norm and the convolution are 32-bit.  A request keeps its last TAPS - 1 rows n in 32-bit, position p in ring row
// p mod (TAPS - 1); rows ahead of position 0 are zero.
//   * conv_norm_row_kernel      one CTA per row: single tokens, and the norm without a convolution;
//   * conv_norm_strip_kernel    one CTA per strip of a portion's rows.  A warp per row takes mean and variance while it streams
//                               the row (chunks of 16 values a lane, merged pairwise, so nothing cancels); then every thread
//                               slides down its own columns, the last TAPS rows n in registers.
// The TAPS - 1 rows in front of a strip are taken once more by it, so strips need nothing from one another, which is also why
// the new residual goes to another buffer.  Strips start at the portion's first row and are at least TAPS - 1 rows long: only
// the first one reads the ring, and it also writes it, taking the portion's last rows itself where they lie in another strip.
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

// Residual columns 4i .. 4i + 3 of a row, with what is added to them.
template <typename T>
struct CnRow {
  const T* embed = nullptr;
  const float* x = nullptr;
  const T* y = nullptr;
  __device__ __forceinline__ CnRow(const ConvNormParams<T>& p, long long row, long long src) {
    if (p.embed) {
      long long tok = p.tokens[row];
      tok = tok < 0 ? 0 : (tok >= p.vocab ? p.vocab - 1 : tok);
      embed = p.embed + tok * p.H;
    } else {
      x = p.x + src * p.H;
    }
    if (p.y) y = p.y + row * p.H;
  }
  __device__ __forceinline__ float4 load(int i, float mult) const {
    float4 v = embed ? ld4(embed + i * 4) : ld4(x + i * 4);
    if (y) {
      const float4 a = ld4(y + i * 4);
      v.x = fmaf(mult, a.x, v.x); v.y = fmaf(mult, a.y, v.y); v.z = fmaf(mult, a.z, v.z); v.w = fmaf(mult, a.w, v.w);
    }
    return v;
  }
};

// v minus the mean, zero in the padding.
__device__ __forceinline__ float4 cn_centred(float4 v, float mean, int c, int H_true) {
  return make_float4(c < H_true ? v.x - mean : 0.f, c + 1 < H_true ? v.y - mean : 0.f, c + 2 < H_true ? v.z - mean : 0.f,
                     c + 3 < H_true ? v.w - mean : 0.f);
}
__device__ __forceinline__ float4 cn_scaled(float4 v, float f, float4 g) {
  return make_float4(v.x * f * g.x, v.y * f * g.y, v.z * f * g.z, v.w * f * g.w);
}
__device__ __forceinline__ void cn_add(float4& o, float4 w, float4 n) {
  o.x = fmaf(w.x, n.x, o.x); o.y = fmaf(w.y, n.y, o.y); o.z = fmaf(w.z, n.z, o.z); o.w = fmaf(w.w, n.w, o.w);
}

// Block-wide sum with one barrier.  Calls alternate between two buffers: a thread that writes one has passed the barrier of the
// call between, so every thread has read what the buffer held.
__device__ __forceinline__ float cn_sum(float a, float (*red)[32], int turn) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffff, a, o);
  float* r = red[turn];
  if (lane == 0) r[w] = a;
  __syncthreads();
  a = lane < nw ? r[lane] : 0.f;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffff, a, o);
  return a;
}

// grid: one CTA per row behind the portions.  Thread i owns the float4 groups i, i + blockDim, ... (NV of them).  TAPS 1: no
// convolution.
template <typename T, int TAPS, int NV>
__global__ void __launch_bounds__(512) conv_norm_row_kernel(const ConvNormParams<T> p) {
  constexpr int W = TAPS - 1, HELD = TAPS > 1 && TAPS <= 4 ? TAPS : 1;
  __shared__ float red[2][32];
  const int tid = threadIdx.x, nv = p.H >> 2;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  // gain and taps are weights: no earlier kernel of the step writes them
  float4 gain[NV], taps[HELD][NV];
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = tid + v * blockDim.x;
    gain[v] = p.gain && i < nv ? ld4(p.gain + i * 4) : zero;
#pragma unroll
    for (int j = 0; j < HELD; ++j)
      taps[j][v] = TAPS > 1 && TAPS <= 4 && i < nv ? ld4(p.taps + static_cast<long long>(j) * p.H + i * 4) : zero;
  }
  auto tap = [&](int j, int v, int i) {
    return TAPS <= 4 ? taps[j < HELD ? j : 0][v] : ld4(p.taps + static_cast<long long>(j) * p.H + i * 4);
  };
  pdl_launch_dependents();
  pdl_wait();
  const long long row = (TAPS > 1 ? p.portion_rows : 0) + static_cast<long long>(blockIdx.x);
  const CnRow<T> src(p, row, TAPS == 1 && p.pick ? p.pick[row] : row);
  const int seg = p.n_portions + blockIdx.x;
  const int pos = TAPS > 1 ? p.first_pos[seg] : 0, slot = TAPS > 1 ? p.states[seg] : -1;
  float* ring = TAPS > 1 ? p.ring + static_cast<long long>(slot < 0 ? 0 : slot) * W * p.H : nullptr;
  float4 x[NV], past[NV];       // past: the earlier rows' part of the convolution
  float s = 0.f;
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = tid + v * blockDim.x;
    x[v] = i < nv ? src.load(i, p.mult) : zero;
    past[v] = zero;
#pragma unroll
    for (int j = 0; j < W; ++j) {
      const int q = pos - W + j;
      const float4 n = i < nv ? ld4(ring + static_cast<long long>((q < 0 ? 0 : q) % (W > 0 ? W : 1)) * p.H + i * 4) : zero;
      cn_add(past[v], tap(j, v, i < nv ? i : 0), q >= 0 && slot >= 0 ? n : zero);
    }
  }
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = tid + v * blockDim.x;
    if (p.x_out && i < nv) st4(p.x_out + row * p.H + i * 4, x[v]);
    s += (x[v].x + x[v].y) + (x[v].z + x[v].w);      // columns past H_true are zero
  }
  if (!p.h) return;
  if (p.center) {
    const float mean = cn_sum(s, red, 0) / p.H_true;
#pragma unroll
    for (int v = 0; v < NV; ++v) x[v] = cn_centred(x[v], mean, (tid + v * blockDim.x) * 4, p.H_true);
  }
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < NV; ++v) ss += sq4(x[v]);
  const float f = 1.f / sqrtf(cn_sum(ss, red, 1) / p.H_true + p.eps);
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = tid + v * blockDim.x;
    if (i >= nv) continue;
    const float4 n = cn_scaled(x[v], f, gain[v]);
    float4 o = n;
    if (TAPS > 1) {
      o = past[v];
      cn_add(o, tap(W, v, i), n);
      if (slot >= 0) st4(ring + static_cast<long long>(pos % (W > 0 ? W : 1)) * p.H + i * 4, n);
    }
    st4(p.h + row * p.H + i * 4, o);
  }
}

constexpr int CS_WARPS = 8;
constexpr int CS_CTAS = 4;                   // resident per SM (up to four taps)
constexpr int CS_AHEAD = 2;                  // rows a thread reads ahead
constexpr int CS_GROUPS = 4;                 // float4 groups a lane takes at a time
constexpr int CS_MAX_ROWS = CS_WARPS * 4;    // rows of a strip and in front of it

// Number, mean and sum of squared deviations of a set, merged with another's.
struct CnMoments {
  float n, mean, m2;
  __device__ __forceinline__ void merge(float nb, float mb, float sb) {
    const float all = n + nb;
    if (nb == 0.f) return;
    const float d = mb - mean, f = nb / all;
    mean = fmaf(d, f, mean);
    m2 += sb + d * d * n * f;
    n = all;
  }
};

// grid: portions x strips.
template <typename T, int TAPS>
__global__ void __launch_bounds__(CS_WARPS * 32, TAPS <= 4 ? CS_CTAS : 2) conv_norm_strip_kernel(const ConvNormParams<T> p) {
  constexpr int W = TAPS - 1;
  __shared__ float s_mean[CS_MAX_ROWS + W], s_rstd[CS_MAX_ROWS + W];   // rows lo - W .. hi - 1, then the portion's last W rows
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nv = p.H >> 2;
  const int seg = blockIdx.x / p.strips, s = blockIdx.x % p.strips;
  const int r_beg = p.cu[seg], r_end = p.cu[seg + 1], lo = r_beg + s * p.strip;
  if (lo >= r_end) return;
  const int hi = lo + p.strip < r_end ? lo + p.strip : r_end;
  const int p0 = p.first_pos[seg], slot = p.states[seg];
  const bool first = s == 0, tail = first && slot >= 0 && hi < r_end;
  const int front = hi - lo + W;             // rows of the first kind
  // row behind index k of the statistics
  auto row_of = [&](int k) { return k < front ? lo - W + k : r_end - W + (k - front); };

  for (int k = warp; k < front + (tail ? W : 0); k += CS_WARPS) {
    const int r = row_of(k);
    if (r < r_beg) continue;                 // it is in the ring, or ahead of the sequence
    const CnRow<T> src(p, r, r);
    const bool store = r >= lo && r < hi && k < front && p.x_out;
    CnMoments m = {0.f, 0.f, 0.f};
    for (int base = 0; base < nv; base += 32 * CS_GROUPS) {
      float4 v[CS_GROUPS];
#pragma unroll
      for (int j = 0; j < CS_GROUPS; ++j) {
        const int i = base + j * 32 + lane;
        v[j] = i < nv ? src.load(i, p.mult) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
      float sum = 0.f, cnt = 0.f;
#pragma unroll
      for (int j = 0; j < CS_GROUPS; ++j) {
        const int i = base + j * 32 + lane, left = p.H_true - i * 4;
        if (store && i < nv) st4(p.x_out + static_cast<long long>(r) * p.H + i * 4, v[j]);
        sum += (v[j].x + v[j].y) + (v[j].z + v[j].w);
        cnt += left >= 4 ? 4.f : left > 0 ? static_cast<float>(left) : 0.f;
      }
      const float mean = p.center && cnt > 0.f ? sum / cnt : 0.f;
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < CS_GROUPS; ++j) ss += sq4(cn_centred(v[j], mean, (base + j * 32 + lane) * 4, p.H_true));
      m.merge(cnt, mean, ss);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float nb = __shfl_xor_sync(0xffffffff, m.n, o), mb = __shfl_xor_sync(0xffffffff, m.mean, o);
      m.merge(nb, mb, __shfl_xor_sync(0xffffffff, m.m2, o));
    }
    if (lane == 0) {
      s_mean[k] = m.mean;
      s_rstd[k] = 1.f / sqrtf(m.m2 / p.H_true + p.eps);
    }
  }
  __syncthreads();                           // also: this CTA's new residual rows are visible to its threads

  for (int i = tid; i < nv; i += CS_WARPS * 32) {
    const float4 gain = ld4(p.gain + i * 4);
    float4 taps[TAPS], win[W];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) taps[j] = ld4(p.taps + static_cast<long long>(j) * p.H + i * 4);
    float* ring = p.ring + static_cast<long long>(slot < 0 ? 0 : slot) * W * p.H + i * 4;
    auto normed = [&](int k, float4 v) { return cn_scaled(cn_centred(v, s_mean[k], i * 4, p.H_true), s_rstd[k], gain); };
#pragma unroll
    for (int j = 0; j < W; ++j) {
      const int r = lo - W + j, q = p0 + (r - r_beg);
      win[j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r >= r_beg) win[j] = normed(j, CnRow<T>(p, r, r).load(i, p.mult));
      else if (q >= 0 && slot >= 0) win[j] = ld4(ring + static_cast<long long>(q % W) * p.H);
    }
    float4 nx[CS_AHEAD];
    auto fetch = [&](int r) {
      if (r >= hi) return make_float4(0.f, 0.f, 0.f, 0.f);
      return p.x_out ? ld4(p.x_out + static_cast<long long>(r) * p.H + i * 4) : CnRow<T>(p, r, r).load(i, p.mult);
    };
#pragma unroll
    for (int a = 0; a < CS_AHEAD; ++a) nx[a] = fetch(lo + a);
    for (int r0 = lo; r0 < hi; r0 += CS_AHEAD) {
      float4 cur[CS_AHEAD];
#pragma unroll
      for (int a = 0; a < CS_AHEAD; ++a) {
        cur[a] = nx[a];
        nx[a] = fetch(r0 + CS_AHEAD + a);       // on their way while these rows are worked on
      }
#pragma unroll
      for (int a = 0; a < CS_AHEAD; ++a) {
        const int r = r0 + a;
        if (r >= hi) break;
        const float4 n = normed(r - lo + W, cur[a]);
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int j = 0; j < W; ++j) cn_add(o, taps[j], win[j]);
        cn_add(o, taps[W], n);
        st4(p.h + static_cast<long long>(r) * p.H + i * 4, o);
#pragma unroll
        for (int j = 0; j + 1 < W; ++j) win[j] = win[j + 1];
        win[W - 1] = n;
      }
    }
    if (first && slot >= 0) {
#pragma unroll
      for (int j = 0; j < W; ++j) {
        const int r = r_end - W + j;
        if (r < r_beg) continue;             // an older row: it is in the ring already
        const float4 n = tail ? normed(front + j, CnRow<T>(p, r, r).load(i, p.mult)) : win[j];
        st4(ring + static_cast<long long>((p0 + (r - r_beg)) % W) * p.H, n);
      }
    }
  }
}

inline int& conv_norm_rounds() {           // > 0: fixed
  static int n = 0;
  return n;
}

template <typename T, int TAPS>
int launch_cn(ConvNormParams<T>& p, int max_portion, cudaStream_t st) {
  if (TAPS > 1 && p.n_portions > 0) {
    // with the rows in front of them, strips make whole rounds of the CTA's warps; the length with the fewest rounds over all
    // waves, one more counted per CTA, and at least W rows
    constexpr int W = TAPS - 1, LEAST = (2 * W + CS_WARPS - 1) / CS_WARPS;
    const long long slots = static_cast<long long>(sm_count()) * (TAPS <= 4 ? CS_CTAS : 2);
    int rounds = LEAST;
    long long best = 1LL << 60;
    for (int n = LEAST; n <= 4; ++n) {
      const int strip = n * CS_WARPS - W;
      const long long ctas = (p.portion_rows + strip - 1) / strip, cost = (ctas + slots - 1) / slots * (n + 1);
      if (cost < best) { best = cost; rounds = n; }
    }
    if (conv_norm_rounds() >= LEAST) rounds = conv_norm_rounds();
    p.strip = rounds * CS_WARPS - W;
    p.strips = (max_portion + p.strip - 1) / p.strip;
    launch_k(conv_norm_strip_kernel<T, (TAPS > 1 ? TAPS : 2)>, dim3(p.n_portions * p.strips), dim3(CS_WARPS * 32), 0, st, p);
  }
  const int single = TAPS > 1 ? p.rows - p.portion_rows : p.rows;
  if (single > 0) {
    const int groups = p.H / 4;
    int per = groups <= 128 ? 1 : 2, threads = ((groups + per - 1) / per + 31) / 32 * 32;
    if (threads > 512) {
      threads = 512;
      per = (groups + threads - 1) / threads;
    }
    const dim3 grid(single), block(threads);
    if (per <= 1) launch_k(conv_norm_row_kernel<T, TAPS, 1>, grid, block, 0, st, p);
    else if (per <= 2) launch_k(conv_norm_row_kernel<T, TAPS, 2>, grid, block, 0, st, p);
    else if (per <= 4) launch_k(conv_norm_row_kernel<T, TAPS, 4>, grid, block, 0, st, p);
    else if (per <= 8) launch_k(conv_norm_row_kernel<T, TAPS, 8>, grid, block, 0, st, p);
    else return -2;
  }
  return launch_status();
}

}  // namespace gk

using namespace gk;

GK_EXPORT void gk_conv_norm_set_rounds(int n) { conv_norm_rounds() = n >= 1 && n <= 4 ? n : 0; }

// ptrs: {tokens, embed, x, y, x_out, gain, taps, ring, cu, first_pos, states, pick, h}
// dims: {rows, H, H_true, n_portions, portion_rows, max_portion, n_taps, vocab, center};  n_taps 0: no convolution, else 2, 3, 4,
// 8 or 16;  H % 4 == 0, H <= 16384.  x_out must not overlap x.  floats: {mult, eps}
GK_EXPORT int gk_conv_norm(int is_fp32, void* const* ptrs, const int* dims, const float* floats, void* stream) {
  const int rows = dims[0], H = dims[1], n_taps = dims[6];
  if (rows == 0) return 0;
  if (rows < 0 || H <= 0 || H % 4 || H > 16384 || dims[2] < 1 || dims[2] > H) return -1;
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
    p.strips = 1; p.strip = 1; p.vocab = dims[7]; p.center = dims[8];
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
