// Routed experts: every token is served by `top` of `experts` small feed-forwards.
//   moe_route    per token (one warp): scores s = sigmoid(z) of the fp32 router logits, or softmax(z) over all
//                experts (`softmax_scores`); the choice is made on
//                s + correction, optionally only among the experts of the `keep` best of `groups` equal groups of
//                neighbours (a group's score: the sum of its two largest choice scores, or its largest alone with
//                `group_max`; experts of other groups
//                count as minus infinity); the weights are the chosen experts' s (divided by their sum + renorm_eps with
//                `renorm`), times `weight_scale`.  Ties go to the lower index.
//                (the logits may come as unsummed splits of their product)
//   moe_align    (one block) sorts the (token, slot) pairs by expert: every expert's pairs form whole tiles of
//                `tile_m` rows (the last one filled up with -1), so that a tile of the products below reads ONE
//                expert's weights; writes the pair of every row, the expert of every tile and the tile count.
//   moe_route_align  both in one launch of one block, for few tokens.
//   moe_gemm     out[pair] = A[row of pair] @ W[expert]^T over the tiles; `gated`: W holds gate and up rows and
//                the result is the gated activation of the two (GateAct: silu(gate) * up, or with a slope, clamps and
//                an offset), rounded to T; `act` 1 (experts without a gate): the square of
//                max(result, 0), rounded to T; otherwise the fp32 result itself.
//   moe_combine  out[token] = sum over its slots, in slot order, of weight * result[pair] (+ a shared expert's
//                result, times sigmoid(shared_gate[token]) when the shared expert has a gate), rounded to T.
// A weight may instead multiply the expert's INPUT (W (w h) = w (W h)): moe_gemm (`row_scale`, one number per pair) and
// the grouped tensor-core product (one per sorted row, filled in by moe_gather) multiply the fp32 accumulators by it
// ahead of the activation, and moe_combine then adds without weights.
// A pair's result does not depend on which other pairs share its tile or on the tile's place: every row is a dot
// product over K in one fixed order.  Scores, choice, weights, accumulators and the combination are fp32.
#include "common.cuh"
#include "row_sum.cuh"
#include <math_constants.h>

#include <algorithm>

namespace {

__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) {
      v = ov;
      i = oi;
    }
  }
}

// Router logits of one product: [n, experts] at `stride`, or up to 16 unsummed splits of it, summed in ascending order.
struct RouterLogits {
  const float* z;
  int64_t stride;
  int n_parts;              // 0: not split
  int64_t part_stride;
  __device__ __forceinline__ float at(int64_t i, int e) const {
    const float* p = z + i * stride + e;
    return n_parts ? sum_parts16(p, n_parts, part_stride) : *p;
  }
};
struct RouteRule {
  int experts, top, groups, keep, renorm, softmax_scores, group_max;
  float renorm_eps, weight_scale;
};

// Token i by one warp; sm: 2 * experts + groups floats of shared memory of this warp's own.
__device__ __forceinline__ void route_token(const RouterLogits& logits, const float* __restrict__ correction,
                                            int* ids, float* weights, int i, const RouteRule& rule, float* sm) {
  const int experts = rule.experts, groups = rule.groups, lane = threadIdx.x & 31;
  float* s = sm;                 // [experts] scores
  float* c = s + experts;        // [experts] choice scores
  float* gs = c + experts;       // [groups] group scores, then 1 = kept
  for (int e = lane; e < experts; e += 32) s[e] = logits.at(i, e);
  float z_max = -CUDART_INF_F, z_sum = 0.f;
  if (rule.softmax_scores) {
    for (int e = lane; e < experts; e += 32) z_max = fmaxf(z_max, s[e]);
    z_max = warp_max(z_max);
    for (int e = lane; e < experts; e += 32) {
      const float v = expf(s[e] - z_max);
      s[e] = v;
      z_sum += v;
    }
    z_sum = warp_sum(z_sum);
  }
  for (int e = lane; e < experts; e += 32) {
    const float v = rule.softmax_scores ? s[e] / z_sum : 1.0f / (1.0f + expf(-s[e]));
    s[e] = v;
    c[e] = v + (correction ? correction[e] : 0.f);
  }
  __syncwarp();
  if (groups > 1 && rule.keep < groups) {
    const int per = experts / groups;
    for (int g = lane; g < groups; g += 32) {
      float m1 = -CUDART_INF_F, m2 = -CUDART_INF_F;
      for (int e = g * per; e < (g + 1) * per; ++e) {
        const float v = c[e];
        if (v > m1) {
          m2 = m1;
          m1 = v;
        } else if (v > m2) {
          m2 = v;
        }
      }
      gs[g] = (per > 1 && !rule.group_max) ? m1 + m2 : m1;
    }
    __syncwarp();
    // the `keep` best groups, one after the other; a kept group is marked by +inf ... then turned into a flag
    for (int r = 0; r < rule.keep; ++r) {
      float best = -CUDART_INF_F;
      int bi = 0x7fffffff;
      for (int g = lane; g < groups; g += 32) {
        const float v = gs[g];
        if (v != CUDART_INF_F && (v > best || bi == 0x7fffffff)) {
          best = v;
          bi = g;
        }
      }
      warp_argmax(best, bi);
      __syncwarp();
      if (lane == 0 && bi < groups) gs[bi] = CUDART_INF_F;
      __syncwarp();
    }
    for (int e = lane; e < experts; e += 32)
      if (gs[e / per] != CUDART_INF_F) c[e] = -CUDART_INF_F;
    __syncwarp();
  }
  float total = 0.f;
  for (int r = 0; r < rule.top; ++r) {
    float best = -CUDART_INF_F;
    int bi = 0x7fffffff;
    for (int e = lane; e < experts; e += 32) {
      const float v = c[e];
      if (v > best) {
        best = v;
        bi = e;
      }
    }
    warp_argmax(best, bi);
    __syncwarp();
    if (bi >= experts) bi = 0;              // nothing left to choose (NaN logits): keep the indices in range
    if (lane == 0) {
      ids[(int64_t)i * rule.top + r] = bi;
      weights[(int64_t)i * rule.top + r] = s[bi];
      c[bi] = -CUDART_INF_F;
    }
    total += s[bi];
    __syncwarp();
  }
  if (rule.renorm || rule.weight_scale != 1.0f) {
    __syncwarp();
    for (int r = lane; r < rule.top; r += 32) {
      float wv = weights[(int64_t)i * rule.top + r];
      if (rule.renorm) wv /= total + rule.renorm_eps;
      weights[(int64_t)i * rule.top + r] = wv * rule.weight_scale;
    }
  }
  __syncwarp();
}

__global__ void __launch_bounds__(32)
moe_route_kernel(RouterLogits logits, const float* __restrict__ correction, int* ids, float* weights, RouteRule rule) {
  extern __shared__ float sm[];
  pdl_trigger();
  pdl_wait();
  route_token(logits, correction, ids, weights, blockIdx.x, rule, sm);
}

// By one block; smi: 3 * experts + 1 ints of shared memory.
__device__ __forceinline__ void align_pairs(const int* ids, int* sorted, int* tile_expert, int* num_tiles, int* row_of_pair,
                                            int n_pairs, int experts, int tile_m, int max_tiles, int* smi) {
  int* counts = smi;                  // [experts]
  int* first = counts + experts;      // [experts + 1] first row of every expert
  int* cursor = first + experts + 1;  // [experts]
  for (int e = threadIdx.x; e < experts; e += blockDim.x) counts[e] = cursor[e] = 0;
  __syncthreads();
  for (int p = threadIdx.x; p < n_pairs; p += blockDim.x) {
    const int e = ids[p];
    if (e >= 0 && e < experts) atomicAdd(&counts[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int at = 0;
    for (int e = 0; e < experts; ++e) {
      first[e] = at;
      at += (counts[e] + tile_m - 1) / tile_m * tile_m;
    }
    first[experts] = at;
    num_tiles[0] = min(at / tile_m, max_tiles);
  }
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += blockDim.x)
    for (int t = first[e] / tile_m; t < first[e + 1] / tile_m && t < max_tiles; ++t) tile_expert[t] = e;
  if (sorted)
    for (int r = threadIdx.x; r < max_tiles * tile_m; r += blockDim.x) sorted[r] = -1;
  __syncthreads();
  for (int p = threadIdx.x; p < n_pairs; p += blockDim.x) {
    const int e = ids[p];
    if (e < 0 || e >= experts) continue;
    const int row = first[e] + atomicAdd(&cursor[e], 1);
    if (sorted && row < max_tiles * tile_m) sorted[row] = p;
    if (row_of_pair) row_of_pair[p] = min(row, max_tiles * tile_m - 1);
  }
}

__global__ void __launch_bounds__(1024)
moe_align_kernel(const int* __restrict__ ids, int* __restrict__ sorted, int* __restrict__ tile_expert,
                 int* __restrict__ num_tiles, int* __restrict__ row_of_pair, int n_pairs, int experts, int tile_m,
                 int max_tiles) {
  extern __shared__ int smi[];
  pdl_trigger();
  pdl_wait();
  align_pairs(ids, sorted, tile_expert, num_tiles, row_of_pair, n_pairs, experts, tile_m, max_tiles, smi);
}

// Both for few tokens, by one block: a warp per token in turn, then the sort.
__global__ void __launch_bounds__(1024)
moe_route_align_kernel(RouterLogits logits, const float* __restrict__ correction, int* ids, float* weights, RouteRule rule,
                       int n_tokens, int* sorted, int* tile_expert, int* num_tiles, int* row_of_pair, int tile_m,
                       int max_tiles) {
  extern __shared__ float sm[];
  pdl_trigger();
  pdl_wait();
  const int per_warp = 2 * rule.experts + rule.groups, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  for (int i = warp; i < n_tokens; i += nwarps) route_token(logits, correction, ids, weights, i, rule, sm + warp * per_warp);
  __syncthreads();
  align_pairs(ids, sorted, tile_expert, num_tiles, row_of_pair, n_tokens * rule.top, rule.experts, tile_m, max_tiles,
              reinterpret_cast<int*>(sm + nwarps * per_warp));
}

// out[row_of_pair[p]] = x[p / top]: the tokens' rows in the order of the sorted pairs (and, with row_scale, the pairs'
// weights in that order), for products that read their rows in place (16 bytes a thread; width * sizeof(T) is a multiple of 16).
template <typename T>
__global__ void __launch_bounds__(256)
moe_gather_kernel(const T* __restrict__ x, int64_t x_stride, const int* __restrict__ row_of_pair, T* __restrict__ out,
                  int top, int width, const float* __restrict__ weights, float* __restrict__ row_scale) {
  pdl_trigger();
  pdl_wait();
  const int p = blockIdx.x;
  if (row_scale && threadIdx.x == 0) row_scale[row_of_pair[p]] = weights[p];
  const uint4* src = reinterpret_cast<const uint4*>(x + (int64_t)(p / top) * x_stride);
  uint4* dst = reinterpret_cast<uint4*>(out + (int64_t)row_of_pair[p] * width);
  const int n16 = width * (int)sizeof(T) / 16;
  for (int i = threadIdx.x; i < n16; i += blockDim.x) dst[i] = src[i];
}

constexpr int MG_M = 16, MG_N = 64, MG_K = 32, MG_THREADS = 128;

// grid (max_tiles, ceil(n_cols / MG_N)).  A row of pair p: a + (p / a_div) * a_stride.  W of expert e: w + e *
// w_expert_stride, rows of k columns; gated: up rows lie `up_offset` elements behind the gate rows.
template <typename T>
__global__ void __launch_bounds__(MG_THREADS)
moe_gemm_kernel(const T* __restrict__ a, int64_t a_stride, int a_div, const T* __restrict__ w, int64_t w_expert_stride,
                int64_t up_offset, const int* __restrict__ sorted, const int* __restrict__ tile_expert,
                const int* __restrict__ num_tiles, T* __restrict__ out_t, float* __restrict__ out_f, int n_cols, int k,
                int act, const float* __restrict__ row_scale, GateAct gate) {
  __shared__ float As[MG_M][MG_K + 1];
  __shared__ float Bs[MG_N][MG_K + 1];
  __shared__ float Us[MG_N][MG_K + 1];
  __shared__ int pairs[MG_M];
  pdl_trigger();
  pdl_wait();
  const int tile = blockIdx.x;
  if (tile >= num_tiles[0]) return;
  const bool gated = up_offset != 0;
  const int tid = threadIdx.x;
  if (tid < MG_M) pairs[tid] = sorted[tile * MG_M + tid];
  __syncthreads();
  const T* we = w + (int64_t)tile_expert[tile] * w_expert_stride;
  const int col0 = blockIdx.y * MG_N;
  const int ty = tid / 16, tx = tid % 16;          // rows 2 ty, 2 ty + 1; columns tx, tx + 16, tx + 32, tx + 48
  float acc[2][4] = {}, acu[2][4] = {};
  for (int k0 = 0; k0 < k; k0 += MG_K) {
    for (int idx = tid; idx < MG_M * MG_K; idx += MG_THREADS) {
      const int r = idx / MG_K, kk = idx % MG_K;
      const int p = pairs[r];
      As[r][kk] = (p >= 0 && k0 + kk < k) ? to_float(a[(int64_t)(p / a_div) * a_stride + k0 + kk]) : 0.f;
    }
    for (int idx = tid; idx < MG_N * MG_K; idx += MG_THREADS) {
      const int c = idx / MG_K, kk = idx % MG_K;
      const bool ok = col0 + c < n_cols && k0 + kk < k;
      const int64_t at = (int64_t)(col0 + c) * k + k0 + kk;
      Bs[c][kk] = ok ? to_float(we[at]) : 0.f;
      if (gated) Us[c][kk] = ok ? to_float(we[up_offset + at]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int kk = 0; kk < MG_K; ++kk) {
      const float a0 = As[2 * ty][kk], a1 = As[2 * ty + 1][kk];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float b = Bs[tx + 16 * j][kk];
        acc[0][j] = fmaf(a0, b, acc[0][j]);
        acc[1][j] = fmaf(a1, b, acc[1][j]);
        if (gated) {
          const float u = Us[tx + 16 * j][kk];
          acu[0][j] = fmaf(a0, u, acu[0][j]);
          acu[1][j] = fmaf(a1, u, acu[1][j]);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int p = pairs[2 * ty + i];
    if (p < 0) continue;
    const float rs = row_scale ? row_scale[p] : 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = col0 + tx + 16 * j;
      if (c >= n_cols) continue;
      if (gated) {
        float g = acc[i][j] * rs, u = acu[i][j] * rs;
        if (gate.limit > 0.f) {
          g = fminf(g, gate.limit);
          u = fminf(fmaxf(u, -gate.limit), gate.limit);
        }
        out_t[(int64_t)p * n_cols + c] = from_float<T>(g / (1.0f + expf(-gate.slope * g)) * (u + gate.offset));
      } else if (act == 1) {
        const float r = fmaxf(acc[i][j] * rs, 0.f);
        out_t[(int64_t)p * n_cols + c] = from_float<T>(r * r);
      } else {
        out_f[(int64_t)p * n_cols + c] = acc[i][j] * rs;
      }
    }
  }
}

// A thread takes VEC neighbouring columns; the rows of up to four slots are requested together.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
moe_combine_kernel(RowSum y, const T* __restrict__ shared, T* __restrict__ out, int width,
                   const float* __restrict__ shared_gate, int64_t shared_gate_stride) {
  pdl_trigger();
  pdl_wait();
  const int64_t t = blockIdx.x;
  const float sg = (shared && shared_gate) ? 1.0f / (1.0f + expf(-shared_gate[t * shared_gate_stride])) : 1.0f;
  for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; c < width; c += gridDim.y * blockDim.x * VEC) {
    float acc[VEC];
    y.sum<VEC>(t, c, width, acc);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      if (shared) acc[e] = fmaf(sg, to_float(shared[t * width + c + e]), acc[e]);
      out[t * width + c + e] = from_float<T>(acc[e]);
    }
  }
}

// out = max(in, 0)^2 rounded to T: the activation of experts without a gate, between the two tensor-core products.
template <typename T>
__global__ void __launch_bounds__(256)
moe_relu_sq_kernel(const float* __restrict__ in, T* __restrict__ out, int64_t n) {
  pdl_trigger();
  pdl_wait();
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const float r = fmaxf(in[i], 0.f);
    out[i] = from_float<T>(r * r);
  }
}

template <typename T>
int moe_gemm_launch(const T* a, int64_t a_stride, int a_div, const T* w, int64_t w_expert_stride, int64_t up_offset,
                    const int* sorted, const int* tile_expert, const int* num_tiles, void* out, int max_tiles,
                    int n_cols, int k, int tile_m, int act, const float* row_scale, GateAct gate, cudaStream_t stream) {
  if (max_tiles <= 0) return 0;
  if (tile_m != MG_M || n_cols < 1 || k < 1 || a_div < 1 || act < 0 || act > 1) return (int)cudaErrorInvalidValue;
  const bool gated = up_offset != 0 || act == 1;
  return gllm_launch(moe_gemm_kernel<T>, dim3(max_tiles, (n_cols + MG_N - 1) / MG_N), dim3(MG_THREADS), 0, stream, a,
                     a_stride, a_div, w, w_expert_stride, up_offset, sorted, tile_expert, num_tiles,
                     gated ? (T*)out : (T*)nullptr, gated ? (float*)nullptr : (float*)out, n_cols, k, act, row_scale,
                     gate);
}
}  // namespace

static bool rule_ok(const RouteRule& r) {
  return r.experts >= 1 && r.top >= 1 && r.top <= r.experts && r.groups >= 1 && r.experts % r.groups == 0 && r.keep >= 1 &&
         r.keep <= r.groups && r.top <= r.keep * (r.experts / r.groups);
}

// logits: [n, experts] at `stride`; n_parts > 0: that many unsummed fp32 splits of it, part_stride floats apart.
GLLM_API int gllm_moe_route(const float* logits, int64_t stride, int n_parts, int64_t part_stride, const float* correction,
                            int* ids, float* weights, int n_tokens, int experts, int top, int groups, int keep, int renorm,
                            int softmax_scores, int group_max, float renorm_eps, float weight_scale,
                            cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  const RouteRule rule{experts, top, groups, keep, renorm, softmax_scores, group_max, renorm_eps, weight_scale};
  const size_t smem = sizeof(float) * (size_t)(2 * experts + groups);
  if (!rule_ok(rule) || n_parts > 16 || smem > 48 * 1024) return (int)cudaErrorInvalidValue;
  return gllm_launch(moe_route_kernel, dim3(n_tokens), dim3(32), smem, stream,
                     RouterLogits{logits, stride, n_parts, part_stride}, correction, ids, weights, rule);
}

GLLM_API int gllm_moe_align(const int* ids, int* sorted, int* tile_expert, int* num_tiles, int* row_of_pair,
                            int n_pairs, int experts, int tile_m, int max_tiles, cudaStream_t stream) {
  if (n_pairs <= 0) return 0;
  const size_t smem = sizeof(int) * (size_t)(3 * experts + 1);
  if (smem > 48 * 1024 || tile_m < 1 || max_tiles < 1) return (int)cudaErrorInvalidValue;
  return gllm_launch(moe_align_kernel, dim3(1), dim3(1024), smem, stream, ids, sorted, tile_expert, num_tiles, row_of_pair,
                     n_pairs, experts, tile_m, max_tiles);
}

// Routing and sorting in one launch of one block, for few tokens (the experts' scores of all warps fit 48 KB).
GLLM_API int gllm_moe_route_align(const float* logits, int64_t stride, int n_parts, int64_t part_stride,
                                  const float* correction, int* ids, float* weights, int n_tokens, int experts, int top,
                                  int groups, int keep, int renorm, int softmax_scores, int group_max, float renorm_eps,
                                  float weight_scale, int* sorted, int* tile_expert, int* num_tiles, int* row_of_pair,
                                  int tile_m, int max_tiles, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  const RouteRule rule{experts, top, groups, keep, renorm, softmax_scores, group_max, renorm_eps, weight_scale};
  const int warps = std::min(32, std::max(4, n_tokens));
  const size_t smem = sizeof(float) * (size_t)warps * (2 * experts + groups) + sizeof(int) * (size_t)(3 * experts + 1);
  if (!rule_ok(rule) || n_parts > 16 || smem > 48 * 1024 || tile_m < 1 || max_tiles < 1) return (int)cudaErrorInvalidValue;
  return gllm_launch(moe_route_align_kernel, dim3(1), dim3(warps * 32), smem, stream,
                     RouterLogits{logits, stride, n_parts, part_stride}, correction, ids, weights, rule, n_tokens, sorted,
                     tile_expert, num_tiles, row_of_pair, tile_m, max_tiles);
}

GLLM_API int gllm_moe_gemm_f32(const float* a, int64_t a_stride, int a_div, const float* w, int64_t w_expert_stride,
                               int64_t up_offset, const int* sorted, const int* tile_expert, const int* num_tiles,
                               void* out, int max_tiles, int n_cols, int k, int tile_m, int act,
                               const float* row_scale, float slope, float limit, float offset, cudaStream_t stream) {
  return moe_gemm_launch<float>(a, a_stride, a_div, w, w_expert_stride, up_offset, sorted, tile_expert, num_tiles, out,
                                max_tiles, n_cols, k, tile_m, act, row_scale, GateAct{slope, limit, offset}, stream);
}
GLLM_API int gllm_moe_gemm_bf16(const __nv_bfloat16* a, int64_t a_stride, int a_div, const __nv_bfloat16* w,
                                int64_t w_expert_stride, int64_t up_offset, const int* sorted, const int* tile_expert,
                                const int* num_tiles, void* out, int max_tiles, int n_cols, int k, int tile_m,
                                int act, const float* row_scale, float slope, float limit, float offset,
                                cudaStream_t stream) {
  return moe_gemm_launch<__nv_bfloat16>(a, a_stride, a_div, w, w_expert_stride, up_offset, sorted, tile_expert,
                                        num_tiles, out, max_tiles, n_cols, k, tile_m, act, row_scale,
                                        GateAct{slope, limit, offset}, stream);
}

template <typename T>
static int moe_combine_launch(const float* y, int n_parts, int64_t part_stride, const float* weights, const T* shared, T* out,
                              const int* row_of_pair, int n_tokens, int top, int width, const float* shared_gate,
                              int64_t shared_gate_stride, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (n_parts < 1 || top < 1 || width < 1) return (int)cudaErrorInvalidValue;
  const RowSum rows{y, n_parts, part_stride, row_of_pair, weights, top};
  const bool vec = width % 4 == 0 && part_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(y) & 15) == 0;
  const int blocks_y = n_tokens >= 64 ? 1 : (width + (vec ? 1024 : 256) - 1) / (vec ? 1024 : 256);
  auto kernel = vec ? moe_combine_kernel<T, 4> : moe_combine_kernel<T, 1>;
  return gllm_launch(kernel, dim3(n_tokens, blocks_y), dim3(256), 0, stream, rows, shared, out, width, shared_gate,
                     shared_gate_stride);
}
// y: [n_parts][rows, width] fp32, the parts added in ascending order first.
#define GLLM_MOE_COMBINE(T, S)                                                                                         \
  GLLM_API int gllm_moe_combine_##S(const float* y, int n_parts, int64_t part_stride, const float* weights,            \
                                    const T* shared, T* out, const int* row_of_pair, int n_tokens, int top, int width, \
                                    const float* shared_gate, int64_t shared_gate_stride, cudaStream_t stream) {       \
    return moe_combine_launch<T>(y, n_parts, part_stride, weights, shared, out, row_of_pair, n_tokens, top, width,     \
                                 shared_gate, shared_gate_stride, stream);                                             \
  }
GLLM_MOE_COMBINE(float, f32)
GLLM_MOE_COMBINE(__nv_bfloat16, bf16)

GLLM_API int gllm_moe_gather_bf16(const __nv_bfloat16* x, int64_t x_stride, const int* row_of_pair, __nv_bfloat16* out,
                                  int n_pairs, int top, int width, const float* weights, float* row_scale,
                                  cudaStream_t stream) {
  if (n_pairs <= 0) return 0;
  if (width % 8 || x_stride % 8 || top < 1 || (reinterpret_cast<uintptr_t>(x) & 15) || (row_scale && !weights))
    return (int)cudaErrorInvalidValue;
  return gllm_launch(moe_gather_kernel<__nv_bfloat16>, dim3(n_pairs), dim3(256), 0, stream, x, x_stride, row_of_pair, out,
                     top, width, weights, row_scale);
}

GLLM_API int gllm_moe_relu_sq_bf16(const float* in, __nv_bfloat16* out, int64_t n, cudaStream_t stream) {
  if (n <= 0) return 0;
  int64_t blocks = (n + 255) / 256;
  if (blocks > (int64_t)gllm_sm_count() * 8) blocks = (int64_t)gllm_sm_count() * 8;
  return gllm_launch(moe_relu_sq_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream, in, out, n);
}
