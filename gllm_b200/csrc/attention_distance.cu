// Softmax attention over the paged cache whose only knowledge of positions is a learned bias by distance:
//     s(i, j) = (q_i . k_j) * scale + bias[h][min(i - j, bias_len - 1)]
//     o_i = sum_j e^s(i,j) v_j / (sum_j e^s(i,j) + e^sink[h])
// over the keys j <= i with i - j < window or j < keep_first (window 0: all of them).  Kernels here:
//   distance_prep       per token: the projections' biases, queries and keys divided by their root mean square per
//                       head (eps inside the root, no weight), values optionally mixed with an earlier layer's values of the same
//                       token; keys and values into their pages, queries into a tensor of their own
//   attention_distance  the attention on the CUDA cores, any widths up to 256 (all of float32)
// Page layout: [kv_heads, block_size, dk] keys, then [kv_heads, block_size, dv] values.  Norms, the mix, scores,
// bias, maxima, sums and accumulators are fp32; keys are taken in blocks of 32 aligned to absolute positions, so a
// result depends neither on how the request was cut into steps nor on the rest of the batch.
#include "common.cuh"
#include <math_constants.h>

namespace {
constexpr int WARPS = 4;
constexpr int MAX_D = 256;

// One warp per (token, head of q, k or v).  The projection rows [q: hq * dk | k: hkv * dk | v: hkv * dv] arrive as a
// tensor or as unsummed fp32 splits (summed in ascending order and rounded to T).  first: [n, hkv * dv] values of
// the first layer that mixes; mode 0: untouched, 1: written, 2: v <- v + lambda * (first - v).
template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
distance_prep_kernel(const T* __restrict__ proj, int64_t stride, const float* __restrict__ parts, int n_parts,
                     int64_t part_stride, const float* __restrict__ bias, float eps, T* __restrict__ q_out,
                     T* __restrict__ first, int mode, float lambda, const int* __restrict__ slot_mapping,
                     T* __restrict__ cache, int n_tokens, int hq, int hkv, int dk, int dv, int block_size,
                     int num_pages, int* __restrict__ status) {
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per_token = hq + 2 * hkv;
  const int64_t item = (int64_t)blockIdx.x * WARPS + warp;
  if (item >= (int64_t)n_tokens * per_token) return;
  const int n = (int)(item / per_token), u = (int)(item - (int64_t)n * per_token);
  const bool is_v = u >= hq + hkv;
  const int width = is_v ? dv : dk;
  const int col = is_v ? (hq + hkv) * dk + (u - hq - hkv) * dv : u * dk;
  const int total = (hq + hkv) * dk + hkv * dv;
  float x[MAX_D / 32], ss = 0.f;
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) {
    const int c = lane + 32 * i;
    x[i] = 0.f;
    if (c < width) {
      x[i] = parts ? to_float(from_float<T>(sum_parts16(parts + (int64_t)n * total + col + c, n_parts, part_stride)))
                   : to_float(proj[(int64_t)n * stride + col + c]);
      if (bias) x[i] += bias[col + c];
      ss = fmaf(x[i], x[i], ss);
    }
  }
  if (!is_v) {
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)dk + eps);
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) x[i] *= inv;
  } else if (mode != 0) {
    T* f = first + (int64_t)n * hkv * dv + (int64_t)(u - hq - hkv) * dv;
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) {
      const int c = lane + 32 * i;
      if (c < dv) {
        if (mode == 1) f[c] = from_float<T>(x[i]);
        else x[i] = (1.0f - lambda) * x[i] + lambda * to_float(f[c]);
      }
    }
  }
  T* dst;
  if (u < hq) {
    dst = q_out + (int64_t)n * hq * dk + (int64_t)u * dk;
  } else {
    const int slot = slot_mapping ? slot_mapping[n] : -1;
    if (slot < 0) return;
    const int page = slot / block_size, off = slot % block_size;
    if (page >= num_pages) {
      if (lane == 0) atomicOr(status, GLLM_STATUS_PAGE_RANGE);
      return;
    }
    T* base = cache + (size_t)page * hkv * block_size * (dk + dv);
    dst = is_v ? base + (size_t)hkv * block_size * dk + ((size_t)(u - hq - hkv) * block_size + off) * dv
               : base + ((size_t)(u - hq) * block_size + off) * dk;
  }
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) {
    const int c = lane + 32 * i;
    if (c < width) dst[c] = from_float<T>(x[i]);
  }
}

// The same for projections that arrive as a tensor, sixteen bytes a lane: `lanes` (a power of two, lanes * VEC >= both
// widths, widths multiples of VEC) neighbouring lanes share a head, so a warp takes 32 / lanes of them.
template <typename T>
__global__ void __launch_bounds__(256)
distance_prep_vec_kernel(const T* __restrict__ proj, int64_t stride, const float* __restrict__ bias, float eps,
                         T* __restrict__ q_out, T* __restrict__ first, int mode, float lambda,
                         const int* __restrict__ slot_mapping, T* __restrict__ cache, int n_tokens, int hq, int hkv,
                         int dk, int dv, int lanes, int block_size, int num_pages, int* __restrict__ status) {
  constexpr int VEC = 16 / sizeof(T);
  pdl_trigger();
  pdl_wait();
  const int sub = threadIdx.x & (lanes - 1);
  const int per_token = hq + 2 * hkv;
  const int64_t item = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) / lanes;
  const bool live = item < (int64_t)n_tokens * per_token;          // (every lane takes part in the shuffles)
  const int n = live ? (int)(item / per_token) : 0, u = live ? (int)(item - (int64_t)n * per_token) : 0;
  const bool is_v = u >= hq + hkv;
  const int width = is_v ? dv : dk, c = sub * VEC;
  const int col = is_v ? (hq + hkv) * dk + (u - hq - hkv) * dv : u * dk;
  const bool mine = live && c < width;
  float x[VEC], ss = 0.f;
#pragma unroll
  for (int e = 0; e < VEC; ++e) x[e] = 0.f;
  if (mine) {
    const uint4 raw = *reinterpret_cast<const uint4*>(proj + (int64_t)n * stride + col + c);
    const T* r = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      x[e] = to_float(r[e]);
      if (bias) x[e] += bias[col + c + e];
      ss = fmaf(x[e], x[e], ss);
    }
  }
  for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!mine) return;
  if (!is_v) {
    const float inv = 1.0f / sqrtf(ss / (float)dk + eps);
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[e] *= inv;
  } else if (mode == 2) {
    const uint4 raw = *reinterpret_cast<const uint4*>(first + (int64_t)n * hkv * dv + (u - hq - hkv) * dv + c);
    const T* f = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[e] = (1.0f - lambda) * x[e] + lambda * to_float(f[e]);
  }
  uint4 packed;
  T* y = reinterpret_cast<T*>(&packed);
#pragma unroll
  for (int e = 0; e < VEC; ++e) y[e] = from_float<T>(x[e]);
  if (is_v && mode == 1) *reinterpret_cast<uint4*>(first + (int64_t)n * hkv * dv + (u - hq - hkv) * dv + c) = packed;
  T* dst;
  if (u < hq) {
    dst = q_out + (int64_t)n * hq * dk + (int64_t)u * dk;
  } else {
    const int slot = slot_mapping ? slot_mapping[n] : -1;
    if (slot < 0) return;
    const int page = slot / block_size, off = slot % block_size;
    if (page >= num_pages) {
      if (sub == 0) atomicOr(status, GLLM_STATUS_PAGE_RANGE);
      return;
    }
    T* base = cache + (size_t)page * hkv * block_size * (dk + dv);
    dst = is_v ? base + (size_t)hkv * block_size * dk + ((size_t)(u - hq - hkv) * block_size + off) * dv
               : base + ((size_t)(u - hq) * block_size + off) * dk;
  }
  *reinterpret_cast<uint4*>(dst + c) = packed;
}

// One warp per (token, query head).
template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
attention_distance_kernel(const T* __restrict__ q, int64_t q_stride, T* __restrict__ out, int64_t out_stride,
                          const T* __restrict__ cache, const int* __restrict__ block_table, int bt_stride,
                          const int* __restrict__ positions, const int* __restrict__ token_row,
                          const float* __restrict__ bias, int bias_len, const float* __restrict__ sink, int n_tokens,
                          int hq, int hkv, int dk, int dv, int block_size, int num_pages, float scale, int window,
                          int keep_first, int* __restrict__ status) {
  __shared__ float q_s[WARPS][MAX_D];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t item = (int64_t)blockIdx.x * WARPS + warp;
  if (item >= (int64_t)n_tokens * hq) return;
  const int n = (int)(item / hq), h = (int)(item - (int64_t)n * hq);
  const int kvh = h / (hq / hkv);
  const int qpos = positions[n];
  const int* bt = block_table + (int64_t)token_row[n] * bt_stride;
  const T* qv = q + (int64_t)n * q_stride + (int64_t)h * dk;
  for (int i = lane; i < dk; i += 32) q_s[warp][i] = to_float(qv[i]);
  __syncwarp();
  const size_t page_elems = (size_t)hkv * block_size * (dk + dv);
  const size_t v_base = (size_t)hkv * block_size * dk;
  const float* b = bias + (int64_t)h * bias_len;
  const int wstart = window > 0 ? max(0, qpos - window + 1) : 0;
  float acc[MAX_D / 32];
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) acc[i] = 0.f;
  float m = sink ? sink[h] : -CUDART_INF_F, l = sink ? 1.f : 0.f;
  for (int j0 = 0; j0 <= qpos; j0 += 32) {
    if (j0 >= keep_first && j0 + 31 < wstart) j0 = wstart & ~31;
    const int j = j0 + lane;
    float s = -CUDART_INF_F;
    int64_t vbase = -1;
    if (j <= qpos && (j >= wstart || j < keep_first)) {
      const int page = bt[j / block_size];
      if (page < 0 || page >= num_pages) {
        atomicOr(status, GLLM_STATUS_PAGE_RANGE);
      } else {
        const int off = j % block_size;
        const T* kp = cache + (size_t)page * page_elems + ((size_t)kvh * block_size + off) * dk;
        float d = 0.f;
        for (int i = 0; i < dk; ++i) d = fmaf(q_s[warp][i], to_float(kp[i]), d);
        s = fmaf(d, scale, b[min(qpos - j, bias_len - 1)]);
        vbase = (int64_t)((size_t)page * page_elems + v_base + ((size_t)kvh * block_size + off) * dv);
      }
    }
    const float m_new = fmaxf(m, warp_max(s));
    if (m_new == -CUDART_INF_F) continue;
    const float p = vbase < 0 ? 0.f : expf(s - m_new);
    const float corr = m == -CUDART_INF_F ? 0.f : expf(m - m_new);
    l = l * corr + warp_sum(p);
    m = m_new;
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) acc[i] *= corr;
    const int count = min(32, qpos - j0 + 1);
    for (int jj = 0; jj < count; ++jj) {
      const float pj = __shfl_sync(0xffffffffu, p, jj);
      const int64_t vb = __shfl_sync(0xffffffffu, vbase, jj);
      if (vb < 0) continue;
      const T* vp = cache + vb;
#pragma unroll
      for (int i = 0; i < MAX_D / 32; ++i) {
        const int c = lane + 32 * i;
        if (c < dv) acc[i] = fmaf(pj, to_float(vp[c]), acc[i]);
      }
    }
  }
  const float inv = l > 0.f ? 1.0f / l : 0.f;
  T* o = out + (int64_t)n * out_stride + (int64_t)h * dv;
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) {
    const int c = lane + 32 * i;
    if (c < dv) o[c] = from_float<T>(acc[i] * inv);
  }
}

template <typename T>
int distance_prep_launch(const T* proj, int64_t stride, const float* parts, int n_parts, int64_t part_stride,
                         const float* bias, float eps, T* q_out, T* first, int mode, float lambda,
                         const int* slot_mapping, T* cache, int n_tokens, int hq, int hkv, int dk, int dv,
                         int block_size, int num_pages, int* status, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (hq <= 0 || hkv <= 0 || dk <= 0 || dk > MAX_D || dv <= 0 || dv > MAX_D || n_parts > 16 ||
      (proj == nullptr) == (parts == nullptr) || (mode != 0 && first == nullptr) ||
      (slot_mapping != nullptr && (block_size <= 0 || cache == nullptr)))
    return (int)cudaErrorInvalidValue;
  constexpr int VEC = 16 / (int)sizeof(T);
  auto odd = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) != 0; };
  if (parts == nullptr && dk % VEC == 0 && dv % VEC == 0 && dk <= 32 * VEC && dv <= 32 * VEC && stride % VEC == 0 &&
      !odd(proj) && !odd(q_out) && !odd(first) && !odd(cache)) {
    int lanes = 1;
    while (lanes * VEC < dk || lanes * VEC < dv) lanes *= 2;
    const int64_t grid = ((int64_t)n_tokens * (hq + 2 * hkv) * lanes + 255) / 256;
    if (grid > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
    return gllm_launch(distance_prep_vec_kernel<T>, dim3((unsigned)grid), dim3(256), 0, stream, proj, stride, bias, eps,
                       q_out, first, mode, lambda, slot_mapping, cache, n_tokens, hq, hkv, dk, dv, lanes, block_size,
                       num_pages, status);
  }
  const int64_t blocks = ((int64_t)n_tokens * (hq + 2 * hkv) + WARPS - 1) / WARPS;
  if (blocks > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  return gllm_launch(distance_prep_kernel<T>, dim3((unsigned)blocks), dim3(WARPS * 32), 0, stream, proj, stride, parts,
                     n_parts, part_stride, bias, eps, q_out, first, mode, lambda, slot_mapping, cache, n_tokens, hq, hkv,
                     dk, dv, block_size, num_pages, status);
}

template <typename T>
int attention_distance_launch(const T* q, int64_t q_stride, T* out, int64_t out_stride, const T* cache,
                              const int* block_table, int bt_stride, const int* positions, const int* token_row,
                              const float* bias, int bias_len, const float* sink, int n_tokens, int hq, int hkv, int dk,
                              int dv, int block_size, int num_pages, float scale, int window, int keep_first,
                              int* status, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (hq <= 0 || hkv <= 0 || hq % hkv || dk <= 0 || dk > MAX_D || dv <= 0 || dv > MAX_D || bias == nullptr ||
      bias_len <= 0 || window < 0 || keep_first < 0 || block_size <= 0)
    return (int)cudaErrorInvalidValue;
  const int64_t blocks = ((int64_t)n_tokens * hq + WARPS - 1) / WARPS;
  if (blocks > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  return gllm_launch(attention_distance_kernel<T>, dim3((unsigned)blocks), dim3(WARPS * 32), 0, stream, q, q_stride, out,
                     out_stride, cache, block_table, bt_stride, positions, token_row, bias, bias_len, sink, n_tokens, hq,
                     hkv, dk, dv, block_size, num_pages, scale, window, keep_first, status);
}
}  // namespace

#define GLLM_DISTANCE_EXPORTS(T, S)                                                                                    \
  GLLM_API int gllm_distance_prep_##S(const T* proj, int64_t stride, const float* parts, int n_parts,                  \
                                      int64_t part_stride, const float* bias, float eps, T* q_out, T* first, int mode, \
                                      float lambda, const int* slot_mapping, T* cache, int n_tokens, int hq, int hkv,  \
                                      int dk, int dv, int block_size, int num_pages, int* status,                      \
                                      cudaStream_t stream) {                                                           \
    return distance_prep_launch<T>(proj, stride, parts, n_parts, part_stride, bias, eps, q_out, first, mode, lambda,   \
                                   slot_mapping, cache, n_tokens, hq, hkv, dk, dv, block_size, num_pages, status,      \
                                   stream);                                                                            \
  }                                                                                                                    \
  GLLM_API int gllm_attention_distance_##S(const T* q, int64_t q_stride, T* out, int64_t out_stride, const T* cache,   \
                                           const int* block_table, int bt_stride, const int* positions,                \
                                           const int* token_row, const float* bias, int bias_len, const float* sink,   \
                                           int n_tokens, int hq, int hkv, int dk, int dv, int block_size,              \
                                           int num_pages, float scale, int window, int keep_first, int* status,        \
                                           cudaStream_t stream) {                                                      \
    return attention_distance_launch<T>(q, q_stride, out, out_stride, cache, block_table, bt_stride, positions,        \
                                        token_row, bias, bias_len, sink, n_tokens, hq, hkv, dk, dv, block_size,        \
                                        num_pages, scale, window, keep_first, status, stream);                         \
  }

GLLM_DISTANCE_EXPORTS(float, f32)
GLLM_DISTANCE_EXPORTS(__nv_bfloat16, bf16)
