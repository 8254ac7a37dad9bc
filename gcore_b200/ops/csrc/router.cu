// Mixture-of-experts routing in one pass per token: softmax or sigmoid scores, optional selection bias, group-limited
// selection (the best `topk_group` of G expert groups by the sum of each group's two best scores), top-k, weight
// normalisation and scaling; and the matching backward from d(weights) to d(logits).
//
// One warp per token, the E scores of a token live in registers (lane l holds experts l, l + 32, ...).  Replaces the
// chain topk / scatter / masked_fill / topk / gather / sum / div of the PyTorch formulation (the semantics of the
// reference's routers: softmax top-k with renormalisation for the Qwen MoE families, sigmoid + bias + node-limited
// groups for the DeepSeek families, gpatch_v4/models/deepseek_v4/modeling_deepseek_v4.py:1120-1219).
// Ties go to the lower expert index.  For few tokens (decode steps) router_fused_kernel computes the logits in the same
// launch, one CTA per token.
#include "host_utils.h"
#include "row_ops.cuh"
#include <cfloat>
#include <stdint.h>

namespace gkr {

constexpr int MAX_K = 16;
constexpr int MAX_G = 32;   // a lane per group

struct RouterParams {
  const float* logits;      // [T, E]
  const float* bias;        // [E] or null (selection only)
  const long long* replay;  // [T, K] or null: forced expert ids
  long long* idx;           // [T, K]
  float* w;                 // [T, K]
  long long T;
  int E, K, G, topk_group;
  int sigmoid, norm;
  float scale;
  long long ld;             // floats between the logits of two tokens
  int* counts;              // [E] or null: tokens of every expert, added to what is there
  int* place;               // [T, K] with counts: the choice's place among its expert's tokens
};

__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
  }
}

// One warp routes token t from its logits in `row`.
template <int VPT>
__device__ __forceinline__ void route_token(const RouterParams& p, long long t, int lane, const float* row) {
  float sc[VPT], sel[VPT];
  // ---- scores (lanes past the last expert hold none)
  if (p.sigmoid) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) sc[i] = lane + 32 * i < p.E ? 1.f / (1.f + expf(-row[lane + 32 * i])) : 0.f;
  } else {
    float m = -FLT_MAX;
#pragma unroll
    for (int i = 0; i < VPT; ++i) { sc[i] = lane + 32 * i < p.E ? row[lane + 32 * i] : -FLT_MAX; m = fmaxf(m, sc[i]); }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) { sc[i] = lane + 32 * i < p.E ? expf(sc[i] - m) : 0.f; s += sc[i]; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    const float inv = 1.f / s;
#pragma unroll
    for (int i = 0; i < VPT; ++i) sc[i] *= inv;
  }
  long long* out_idx = p.idx + t * p.K;
  float* out_w = p.w + t * p.K;
  float chosen_w[MAX_K];
  int chosen_i[MAX_K];
  if (p.replay) {
#pragma unroll
    for (int k = 0; k < MAX_K; ++k) {
      if (k >= p.K) break;
      const int e = static_cast<int>(p.replay[t * p.K + k]);
      float v = 0.f;
#pragma unroll
      for (int i = 0; i < VPT; ++i)
        if (lane + 32 * i == e) v = sc[i];
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      chosen_w[k] = v;
      chosen_i[k] = e;
    }
  } else {
#pragma unroll
    for (int i = 0; i < VPT; ++i)
      sel[i] = lane + 32 * i < p.E ? sc[i] + (p.bias ? p.bias[lane + 32 * i] : 0.f) : -FLT_MAX;
    if (p.G > 1) {
      // group score = sum of the two best selection scores inside the group (of the only one in a group of one)
      const int gs = p.E / p.G;
      float mine = -FLT_MAX;               // lane g: score of group g
      for (int g = 0; g < p.G; ++g) {
        float a = -FLT_MAX, b = -FLT_MAX;  // a >= b
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          if ((lane + 32 * i) / gs == g) {
            const float v = sel[i];
            if (v > a) { b = a; a = v; } else if (v > b) { b = v; }
          }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
          const float oa = __shfl_xor_sync(0xffffffffu, a, o), ob = __shfl_xor_sync(0xffffffffu, b, o);
          const float na = fmaxf(a, oa);
          const float nb = fmaxf(fminf(a, oa), fmaxf(b, ob));
          a = na; b = nb;
        }
        if (lane == g) mine = gs > 1 ? a + b : a;
      }
      int rank = 0;
      for (int g = 0; g < p.G; ++g) {
        const float other = __shfl_sync(0xffffffffu, mine, g);
        rank += (other > mine || (other == mine && g < lane)) ? 1 : 0;
      }
      const unsigned kept = __ballot_sync(0xffffffffu, lane < p.G && rank < p.topk_group);
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int g = (lane + 32 * i) / gs;
        if (g >= p.G || !((kept >> g) & 1u)) sel[i] = -FLT_MAX;
      }
    }
#pragma unroll
    for (int k = 0; k < MAX_K; ++k) {
      if (k >= p.K) break;
      float bv = -FLT_MAX;
      int bi = 1 << 30;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        // strict > keeps the lowest index among a lane's equal values (indices grow with i)
        if (sel[i] > bv) { bv = sel[i]; bi = lane + 32 * i; }
      }
      if (bv == -FLT_MAX) bi = 1 << 30;
      float v = bv;
      int e = bi;
      warp_argmax(v, e);
      if (e >= p.E) e = k < p.E ? k : 0;  // fewer selectable experts than K: cannot happen with valid configurations
      float cw = 0.f;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        if (lane + 32 * i == e) { cw = sc[i]; sel[i] = -FLT_MAX; }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) cw += __shfl_xor_sync(0xffffffffu, cw, o);
      chosen_w[k] = cw;
      chosen_i[k] = e;
    }
  }
  float denom = 1.f;
  if (p.norm) {
    denom = 0.f;
#pragma unroll
    for (int k = 0; k < MAX_K; ++k)
      if (k < p.K) denom += chosen_w[k];
    denom = fmaxf(denom, 1e-20f);
  }
  if (lane < p.K) {
    // every lane holds all K results; lane k writes entry k
    float wv = 0.f;
    int iv = 0;
#pragma unroll
    for (int k = 0; k < MAX_K; ++k)
      if (k == lane) { wv = chosen_w[k]; iv = chosen_i[k]; }
    out_idx[lane] = iv;
    out_w[lane] = wv / denom * p.scale;
    if (p.counts) p.place[t * p.K + lane] = atomicAdd(p.counts + iv, 1);
  }
}

template <int VPT>
__global__ void __launch_bounds__(256) router_fwd_kernel(RouterParams p) {
  const long long t = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  gk::pdl_launch_dependents();
  gk::pdl_wait();
  if (t >= p.T) return;
  route_token<VPT>(p, t, threadIdx.x & 31, p.logits + t * p.ld);
}

constexpr int RF_WARPS = 16;
constexpr int RF_MAX_ROWS = 516;

// logits[t, r] = h[t] . w[r] for the `n_rows` rows of w (the experts, then rows the router only projects), then the
// choice among the first E.  H is a multiple of 8.
template <typename T, int VPT>
__global__ void __launch_bounds__(RF_WARPS * 32) router_fused_kernel(RouterParams p, const T* __restrict__ h,
                                                                     const T* __restrict__ w, float* __restrict__ logits,
                                                                     int H, int n_rows) {
  extern __shared__ float rf_h[];
  __shared__ float s_logit[RF_MAX_ROWS];
  gk::pdl_launch_dependents();
  gk::pdl_wait();
  const long long t = blockIdx.x;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  for (int d = tid * 4; d < H; d += RF_WARPS * 128) gk::st4(rf_h + d, gk::ld4(h + t * H + d));
  __syncthreads();
  for (int r0 = warp * 4; r0 < n_rows; r0 += RF_WARPS * 4) {      // four rows at a time: their loads overlap
    float a[4] = {0.f, 0.f, 0.f, 0.f};
    const T* wr[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) wr[i] = w + static_cast<long long>(r0 + i < n_rows ? r0 + i : n_rows - 1) * H;
#pragma unroll 2
    for (int d = lane * 4; d < H; d += 128) {
      const float4 x = gk::ld4(rf_h + d);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 y = gk::ld4(wr[i] + d);
        a[i] = fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, fmaf(x.w, y.w, a[i]))));
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) a[i] += __shfl_xor_sync(0xffffffffu, a[i], o);
      if (lane == 0 && r0 + i < n_rows) {
        s_logit[r0 + i] = a[i];
        logits[t * n_rows + r0 + i] = a[i];
      }
    }
  }
  __syncthreads();
  if (warp == 0) route_token<VPT>(p, t, lane, s_logit);
}

struct RouterBwdParams {
  const float* logits;     // [T, E]
  const long long* idx;    // [T, K]
  const float* dw;         // [T, K]
  float* dlogits;          // [T, E]
  long long T;
  int E, K, sigmoid, norm;
  float scale;
};

template <int VPT>
__global__ void __launch_bounds__(256) router_bwd_kernel(RouterBwdParams p) {
  const long long t = (blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (t >= p.T) return;
  const float* row = p.logits + t * p.E;
  float sc[VPT], g[VPT];
  if (p.sigmoid) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) sc[i] = 1.f / (1.f + expf(-row[lane + 32 * i]));
  } else {
    float m = -FLT_MAX;
#pragma unroll
    for (int i = 0; i < VPT; ++i) { sc[i] = row[lane + 32 * i]; m = fmaxf(m, sc[i]); }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) { sc[i] = expf(sc[i] - m); s += sc[i]; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    const float inv = 1.f / s;
#pragma unroll
    for (int i = 0; i < VPT; ++i) sc[i] *= inv;
  }
  // gradient w.r.t. the selected scores: w_k = scale * s_k / S (S = sum of selected scores, or 1 without normalisation)
#pragma unroll
  for (int i = 0; i < VPT; ++i) g[i] = 0.f;
  float S = 0.f, dot = 0.f;  // S = sum_k s_k,  dot = sum_k dw_k s_k
  for (int k = 0; k < p.K; ++k) {
    const int e = static_cast<int>(p.idx[t * p.K + k]);
    const float d = p.dw[t * p.K + k];
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i)
      if (lane + 32 * i == e) { v = sc[i]; g[i] += d; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    S += v;
    dot += d * v;
  }
  if (p.norm) {
    S = fmaxf(S, 1e-20f);
    const float c = p.scale / S, shift = dot / S;
    for (int k = 0; k < p.K; ++k) {
      const int e = static_cast<int>(p.idx[t * p.K + k]);
#pragma unroll
      for (int i = 0; i < VPT; ++i)
        if (lane + 32 * i == e) g[i] -= shift;  // once per occurrence of the expert in the list
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i) g[i] *= c;
  } else {
#pragma unroll
    for (int i = 0; i < VPT; ++i) g[i] *= p.scale;
  }
  float* out = p.dlogits + t * p.E;
  if (p.sigmoid) {
#pragma unroll
    for (int i = 0; i < VPT; ++i) out[lane + 32 * i] = g[i] * sc[i] * (1.f - sc[i]);
  } else {
    float gp = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) gp += g[i] * sc[i];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) gp += __shfl_xor_sync(0xffffffffu, gp, o);
#pragma unroll
    for (int i = 0; i < VPT; ++i) out[lane + 32 * i] = sc[i] * (g[i] - gp);
  }
}

template <typename P, typename F>
int dispatch_vpt(int E, const P& p, F launch) {
  if (E <= 32) return launch(std::integral_constant<int, 1>{});
  if (E <= 64) return launch(std::integral_constant<int, 2>{});
  if (E <= 128) return launch(std::integral_constant<int, 4>{});
  if (E <= 256) return launch(std::integral_constant<int, 8>{});
  if (E <= 512) return launch(std::integral_constant<int, 16>{});
  return -2;
}

}  // namespace gkr

using namespace gkr;

static bool router_valid(const RouterParams& p) {
  return p.E >= 1 && p.K >= 1 && p.K <= MAX_K && p.K <= p.E && p.G >= 1 && p.G <= MAX_G && p.E % p.G == 0 &&
         (p.G == 1 || (p.topk_group >= 1 && p.topk_group <= p.G));
}

static int router_launch(const RouterParams& p, cudaStream_t st) {
  if (!router_valid(p)) return -1;
  const unsigned blocks = static_cast<unsigned>((p.T + 7) / 8);
  return dispatch_vpt(p.E, p, [&](auto v) {
    gk::launch_k(router_fwd_kernel<decltype(v)::value>, dim3(blocks), dim3(256), 0, st, p);
    return gk::launch_status();
  });
}

// E <= 512; K <= 16; G <= 32 and E % G == 0.  Returns -2 for an expert count without a kernel.
GK_EXPORT int gk_router_fwd(const float* logits, const float* bias, const long long* replay, long long* idx, float* w,
                            long long T, int E, int K, int G, int topk_group, int sigmoid, int norm, float scale,
                            void* stream) {
  if (T <= 0) return 0;
  RouterParams p;
  p.logits = logits; p.bias = bias; p.replay = replay; p.idx = idx; p.w = w; p.T = T; p.E = E; p.K = K; p.G = G;
  p.topk_group = topk_group; p.sigmoid = sigmoid; p.norm = norm; p.scale = scale;
  p.ld = E; p.counts = nullptr; p.place = nullptr;
  return router_launch(p, reinterpret_cast<cudaStream_t>(stream));
}

// Routing of served models: logits rows `ld` floats apart, and the dispatch bookkeeping in the same launch (counts [E],
// cleared by the caller, and every choice's place [T, K] among its expert's tokens; the places' order is not fixed).
GK_EXPORT int gk_router_dispatch(const float* logits, long long ld, const float* bias, long long* idx, float* w, int* counts,
                                 int* place, long long T, int E, int K, int sigmoid, int norm, float scale, int G,
                                 int topk_group, void* stream) {
  if (T <= 0) return 0;
  if (ld < E || !counts || !place) return -1;
  RouterParams p;
  p.logits = logits; p.bias = bias; p.replay = nullptr; p.idx = idx; p.w = w; p.T = T; p.E = E; p.K = K; p.G = G;
  p.topk_group = topk_group; p.sigmoid = sigmoid; p.norm = norm; p.scale = scale;
  p.ld = ld; p.counts = counts; p.place = place;
  return router_launch(p, reinterpret_cast<cudaStream_t>(stream));
}

// The same from the tokens themselves, h [T, H] and w [n_rows, H] (n_rows >= E; H % 8 == 0, at most 11264): also writes the
// logits [T, n_rows].
GK_EXPORT int gk_router_fused(int is_fp32, const void* h, const void* w, float* logits, int H, int n_rows, const float* bias,
                              long long* idx, float* weight, int* counts, int* place, long long T, int E, int K, int sigmoid,
                              int norm, float scale, int G, int topk_group, void* stream) {
  if (T <= 0) return 0;
  if (n_rows < E || n_rows > RF_MAX_ROWS || H % 8 || H > 11264 || !counts || !place) return -1;
  RouterParams p;
  p.logits = logits; p.bias = bias; p.replay = nullptr; p.idx = idx; p.w = weight; p.T = T; p.E = E; p.K = K; p.G = G;
  p.topk_group = topk_group; p.sigmoid = sigmoid; p.norm = norm; p.scale = scale;
  p.ld = n_rows; p.counts = counts; p.place = place;
  if (!router_valid(p)) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return dispatch_vpt(E, p, [&](auto v) {
    constexpr int VPT = decltype(v)::value;
    const dim3 grid(static_cast<unsigned>(T)), block(RF_WARPS * 32);
    if (is_fp32)
      gk::launch_k(router_fused_kernel<float, VPT>, grid, block, H * sizeof(float), st, p, static_cast<const float*>(h),
                   static_cast<const float*>(w), logits, H, n_rows);
    else
      gk::launch_k(router_fused_kernel<__nv_bfloat16, VPT>, grid, block, H * sizeof(float), st, p,
                   static_cast<const __nv_bfloat16*>(h), static_cast<const __nv_bfloat16*>(w), logits, H, n_rows);
    return gk::launch_status();
  });
}

GK_EXPORT int gk_router_bwd(const float* logits, const long long* idx, const float* dw, float* dlogits, long long T,
                            int E, int K, int sigmoid, int norm, float scale, void* stream) {
  if (T <= 0) return 0;
  if (E % 32 || K < 1 || K > MAX_K) return -1;
  RouterBwdParams p;
  p.logits = logits; p.idx = idx; p.dw = dw; p.dlogits = dlogits; p.T = T; p.E = E; p.K = K; p.sigmoid = sigmoid;
  p.norm = norm; p.scale = scale;
  const unsigned blocks = static_cast<unsigned>((T + 7) / 8);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return dispatch_vpt(E, p, [&](auto v) {
    router_bwd_kernel<decltype(v)::value><<<blocks, 256, 0, st>>>(p);
    return gk::launch_status();
  });
}
