// What stands between two sublayers of a layer that norms a sublayer's RESULT and lets the next sublayer read the
// residual itself, convolved over time, with the residual optionally averaged over the depth of the model:
//   X[t] = resid[t] + rms(value[t] + value_bias) * post_w          a sublayer's result joins the residual
//   x[t] = sum_j depth_w[j] * X_j[t]                               (at a layer's end) over the embedding output, every
//                                                                  earlier layer's result and X itself
//   out[t] = x[t] + sum_j conv_w[j] * x[t - taps + 1 + j]          a causal convolution per channel, zeros before the
//                                                                  sequence's start, earlier inputs from `conv_state`
// in one kernel (depth_conv), and the same without the convolution but with an RMS norm of x at chosen rows for the
// model's output (depth_norm).  `value` may arrive as unsummed fp32 splits of a product (summed in ascending order
// and rounded to T first).  Everything is fp32 but `value` and `out`.
//
// A block takes CHUNK consecutive tokens of one request.  Rows before them that the convolution reaches into belong to
// another block, which writes them; this block computes them again (the inputs are not written in place, so there is
// no order between blocks).  The first block of a request reads the request's state and is also the one that brings
// it up to date: it computes the request's last taps-1 rows again when they are not its own.
#include "common.cuh"
#include <algorithm>

namespace {
constexpr int MAX_TAPS = 16;
constexpr int ROWS_MAX = 48;
constexpr int THREADS_MAX = 512;
constexpr int CHUNK = 8;                 // tokens per block

template <int VEC> __device__ __forceinline__ void ld(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
  } else {
    v[0] = p[0];
  }
}
template <int VEC> __device__ __forceinline__ void ld(const __nv_bfloat16* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = lo.x, v[1] = lo.y, v[2] = hi.x, v[3] = hi.y;
  } else {
    v[0] = __bfloat162float(p[0]);
  }
}
template <int VEC> __device__ __forceinline__ void st(float* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else p[0] = v[0];
}
template <int VEC> __device__ __forceinline__ void st(__nv_bfloat16* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    uint2 raw;
    *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v[0], v[1]);
    *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = raw;
  } else {
    p[0] = __float2bfloat16_rn(v[0]);
  }
}

// What joins the residual, and the streams of the depth average.
template <typename T>
struct Joined {
  const T* value;            // [n, width] or null
  const float* parts;        // [n_parts][n, width] or null
  int n_parts;
  int64_t part_stride;
  const float* value_bias;   // [width] or null: the bias of the product that made value
  const float* post_w;       // [width]
  float post_eps;
  const float* resid;        // [n, width]
  float* streams;            // [count + 1][n, width]: X_0 .. X_(count-1), place for X_count; null: no average
  int64_t stream_stride;
  int count;
  const float* depth_w;      // [count + 1] or null
};

// VEC columns of value[row] + bias (from xs when the row was staged there).
template <typename T, int VEC>
__device__ __forceinline__ void joined_value(const Joined<T>& j, const float* staged, int64_t at, int c, float (&v)[VEC]) {
  if (staged) {
    ld<VEC>(staged + c, v);
    return;
  }
  ld<VEC>(j.value + at + c, v);
  if (j.value_bias) {
    float b[VEC];
    ld<VEC>(j.value_bias + c, b);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] += b[e];
  }
}

// Sums the splits of one row into xs (with the bias), columns c = first, first + stride, ...
template <typename T, int VEC>
__device__ __forceinline__ float stage_row(const Joined<T>& j, float* xs, int64_t at, int width, int first, int stride) {
  float ss = 0.f;
  for (int c = first; c < width; c += stride) {
    float v[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      v[e] = to_float(from_float<T>(sum_parts16(j.parts + at + c + e, j.n_parts, j.part_stride)));
      if (j.value_bias) v[e] += j.value_bias[c + e];
      ss = fmaf(v[e], v[e], ss);
    }
    st<VEC>(xs + c, v);
  }
  return ss;
}

template <typename T, int VEC>
__device__ __forceinline__ float row_squares(const Joined<T>& j, int64_t at, int width, int first, int stride) {
  float ss = 0.f;
#pragma unroll 8
  for (int c = first; c < width; c += stride) {
    float v[VEC];
    joined_value<T, VEC>(j, nullptr, at, c, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(v[e], v[e], ss);
  }
  return ss;
}

// What one row's VEC columns bring: the residual, the sublayer's result, the weighted sum of the earlier streams.
template <int VEC>
struct RowIn {
  float r[VEC], v[VEC], s[VEC];
};
template <typename T, int VEC>
__device__ __forceinline__ void fetch_row(const Joined<T>& j, const float* staged, int64_t at, int c, bool has_value,
                                          RowIn<VEC>& in) {
  ld<VEC>(j.resid + at + c, in.r);
  if (has_value) joined_value<T, VEC>(j, staged, at, c, in.v);
  if (j.depth_w) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) in.s[e] = 0.f;
#pragma unroll 4
    for (int k = 0; k < j.count; ++k) {
      float s[VEC];
      ld<VEC>(j.streams + (int64_t)k * j.stream_stride + at + c, s);
      const float w = j.depth_w[k];
#pragma unroll
      for (int e = 0; e < VEC; ++e) in.s[e] = fmaf(w, s[e], in.s[e]);
    }
  }
}
// X and x from it.
template <typename T, int VEC>
__device__ __forceinline__ void joined_x(const Joined<T>& j, const RowIn<VEC>& in, float inv, bool has_value,
                                         const float (&pw)[VEC], float (&X)[VEC], float (&x)[VEC]) {
#pragma unroll
  for (int e = 0; e < VEC; ++e) X[e] = has_value ? fmaf(in.v[e] * inv, pw[e], in.r[e]) : in.r[e];
  if (j.depth_w) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[e] = in.s[e];
    const float w = j.depth_w[j.count];
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[e] = fmaf(w, X[e], x[e]);
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[e] = X[e];
  }
}

// conv_w: [taps, width], the last row multiplies the current token; conv_state: [slots, taps-1, width], oldest first.
// TMAX >= taps: the window a thread keeps (what lies beyond `taps` is multiplied by zero).
template <typename T, int TMAX, int VEC>
__global__ void __launch_bounds__(THREADS_MAX)
depth_conv_kernel(Joined<T> j, float* __restrict__ x_out, const float* __restrict__ conv_w, float* __restrict__ conv_state,
                  const int* __restrict__ cu_q, const int* __restrict__ state_slots, T* __restrict__ out, int width,
                  int taps, int chunk) {
  extern __shared__ __align__(16) float xs[];
  __shared__ float scratch[32];
  __shared__ float inv_s[ROWS_MAX];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.y, keep = taps - 1;
  const int t0 = cu_q[r], len = cu_q[r + 1] - t0;
  const int begin = blockIdx.x * chunk;
  if (begin >= len) return;
  const bool opens = blockIdx.x == 0;
  const int end = min(begin + chunk, len);
  const int first_row = opens ? 0 : begin - keep;          // chunk >= keep
  const int own = end - first_row;
  // the request's last rows, computed again for the state
  const int tail = opens ? max(end, len - keep) : len;
  const int count = own + (len - tail);
  const bool has_value = j.value != nullptr || j.parts != nullptr;
  const int first = threadIdx.x * VEC, stride = blockDim.x * VEC;
  auto row_of = [&](int i) { return i < own ? first_row + i : tail + (i - own); };
  if (has_value) {
    if (j.parts || count < 3) {
      for (int i = 0; i < count; ++i) {
        const int64_t at = (int64_t)(t0 + row_of(i)) * width;
        const float ss = j.parts ? stage_row<T, VEC>(j, xs + (int64_t)i * width, at, width, first, stride)
                                 : row_squares<T, VEC>(j, at, width, first, stride);
        const float total = block_sum(ss, scratch);
        if (threadIdx.x == 0) inv_s[i] = 1.0f / sqrtf(total / (float)width + j.post_eps);
      }
    } else {
      const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
      for (int i = warp; i < count; i += nwarps) {
        const float total =
            warp_sum(row_squares<T, VEC>(j, (int64_t)(t0 + row_of(i)) * width, width, lane * VEC, 32 * VEC));
        if (lane == 0) inv_s[i] = 1.0f / sqrtf(total / (float)width + j.post_eps);
      }
    }
    __syncthreads();
  }
  float* cs = conv_state + (int64_t)state_slots[r] * keep * width;
  for (int c = first; c < width; c += stride) {
    float pw[VEC] = {}, wt[TMAX][VEC], win[TMAX][VEC];      // win[TMAX - 1]: the current row
    if (has_value) ld<VEC>(j.post_w + c, pw);
#pragma unroll
    for (int k = 0; k < TMAX; ++k)
#pragma unroll
      for (int e = 0; e < VEC; ++e) wt[k][e] = win[k][e] = 0.f;
#pragma unroll
    for (int k = 0; k < TMAX; ++k) {
      const int tap = k - (TMAX - taps);
      if (tap >= 0) {
        ld<VEC>(conv_w + (int64_t)tap * width + c, wt[k]);
        // entry tap of the state is what the window holds just before the first row comes in
        if (opens && tap < keep) ld<VEC>(cs + (int64_t)tap * width + c, win[k + 1 < TMAX ? k + 1 : k]);
      }
    }
    // a row's loads are issued a row ahead, before the stores of the row in hand
    auto fetch = [&](int i, RowIn<VEC>& in) {
      fetch_row<T, VEC>(j, j.parts ? xs + (int64_t)i * width : nullptr, (int64_t)(t0 + row_of(i)) * width, c, has_value, in);
    };
    RowIn<VEC> now, next;
    fetch(0, now);
    for (int i = 0; i < count; ++i, now = next) {
      if (i + 1 < count) fetch(i + 1, next);
      const int row = row_of(i);
      const int64_t at = (int64_t)(t0 + row) * width;
      float X[VEC], x[VEC];
      joined_x<T, VEC>(j, now, has_value ? inv_s[i] : 0.f, has_value, pw, X, x);
#pragma unroll
      for (int k = 0; k + 1 < TMAX; ++k)
#pragma unroll
        for (int e = 0; e < VEC; ++e) win[k][e] = win[k + 1][e];
#pragma unroll
      for (int e = 0; e < VEC; ++e) win[TMAX - 1][e] = x[e];
      if (i >= own || row < begin) continue;
      if (j.depth_w) st<VEC>(j.streams + (int64_t)j.count * j.stream_stride + at + c, X);
      if (x_out) st<VEC>(x_out + at + c, x);
      float h[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) h[e] = 0.f;
#pragma unroll
      for (int k = 0; k < TMAX; ++k)
#pragma unroll
        for (int e = 0; e < VEC; ++e) h[e] = fmaf(wt[k][e], win[k][e], h[e]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) h[e] += x[e];
      st<VEC>(out + at + c, h);
    }
    if (opens) {
#pragma unroll
      for (int k = 0; k < TMAX; ++k) {
        const int tap = k - (TMAX - taps);                   // win[k] is input `tap` of the last `taps`; the newest keep stay
        if (tap >= 1) st<VEC>(cs + (int64_t)(tap - 1) * width + c, win[k]);
      }
    }
  }
}

// One block per wanted row: out = rms(x) * w.
template <typename T, int VEC>
__global__ void __launch_bounds__(512)
depth_norm_kernel(Joined<T> j, const int* __restrict__ rows, const float* __restrict__ w, float eps, T* __restrict__ out,
                  int width) {
  extern __shared__ __align__(16) float xs[];
  __shared__ float scratch[32];
  pdl_trigger();
  pdl_wait();
  const int64_t at = (int64_t)(rows ? rows[blockIdx.x] : (int)blockIdx.x) * width;
  const bool has_value = j.value != nullptr || j.parts != nullptr;
  const int first = threadIdx.x * VEC, stride = blockDim.x * VEC;
  float inv = 0.f;
  if (has_value) {
    const float ss = j.parts ? stage_row<T, VEC>(j, xs, at, width, first, stride)
                             : row_squares<T, VEC>(j, at, width, first, stride);
    inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + j.post_eps);
  }
  float ss = 0.f;
  for (int c = first; c < width; c += stride) {
    float pw[VEC] = {}, X[VEC], x[VEC];
    RowIn<VEC> in;
    if (has_value) ld<VEC>(j.post_w + c, pw);
    fetch_row<T, VEC>(j, j.parts ? xs : nullptr, at, c, has_value, in);
    joined_x<T, VEC>(j, in, inv, has_value, pw, X, x);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(x[e], x[e], ss);
    st<VEC>(xs + c, x);                                      // read back by the thread that wrote it
  }
  const float scale = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
  T* o = out + (int64_t)blockIdx.x * width;
  for (int c = first; c < width; c += stride) {
    float v[VEC], ww[VEC];
    ld<VEC>((const float*)xs + c, v);
    ld<VEC>(w + c, ww);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = v[e] * scale * ww[e];
    st<VEC>(o + c, v);
  }
}

inline bool odd(const void* p) { return p != nullptr && (reinterpret_cast<uintptr_t>(p) & 15) != 0; }

template <typename T>
bool four_columns(const Joined<T>& j, int width) {
  return width % 4 == 0 && j.stream_stride % 4 == 0 && !odd(j.value) && !odd(j.parts) && !odd(j.value_bias) &&
         !odd(j.post_w) && !odd(j.resid) && !odd(j.streams);
}

template <typename T>
bool valid(const Joined<T>& j, int width) {
  return width > 0 && j.resid != nullptr && j.n_parts <= 16 && (j.value == nullptr || j.parts == nullptr) &&
         ((j.value == nullptr && j.parts == nullptr) || j.post_w != nullptr) &&
         (j.depth_w == nullptr || (j.streams != nullptr && j.count >= 0));
}

inline int threads_for(int width, int vec) {
  return std::max(32, std::min(THREADS_MAX, (width / vec + 31) / 32 * 32));
}

template <typename K>
int allow_smem(K kernel, size_t smem) {
  if (smem <= 48 * 1024) return 0;
  return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

template <typename T>
int depth_conv_launch(Joined<T> j, float* x_out, const float* conv_w, float* conv_state, const int* cu_q,
                      const int* state_slots, T* out, int num_requests, int max_q_len, int width, int taps,
                      cudaStream_t stream) {
  if (num_requests <= 0 || max_q_len <= 0) return 0;
  if (!valid(j, width) || taps < 1 || taps > MAX_TAPS || num_requests > 65535 || conv_w == nullptr || out == nullptr ||
      (taps > 1 && conv_state == nullptr) || x_out == j.resid)
    return (int)cudaErrorInvalidValue;
  const int chunk = max_q_len == 1 ? std::max(1, taps - 1) : std::max(CHUNK, taps - 1);
  const int rows_most = max_q_len == 1 ? 1 : chunk + taps - 1;
  const size_t smem = j.parts ? sizeof(float) * (size_t)rows_most * width : 0;
  if (rows_most > ROWS_MAX || smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  const bool vec = taps <= 4 && four_columns(j, width) && !odd(x_out) && !odd(conv_w) && !odd(conv_state) && !odd(out);
  auto kernel = vec ? depth_conv_kernel<T, 4, 4> : (taps <= 4 ? depth_conv_kernel<T, 4, 1> : depth_conv_kernel<T, 16, 1>);
  if (int e = allow_smem(kernel, smem)) return e;
  return gllm_launch(kernel, dim3((max_q_len + chunk - 1) / chunk, num_requests), dim3(threads_for(width, vec ? 4 : 1)),
                     smem, stream, j, x_out, conv_w, conv_state, cu_q, state_slots, out, width, taps, chunk);
}

template <typename T>
int depth_norm_launch(Joined<T> j, const int* rows, int n_rows, const float* w, float eps, T* out, int width,
                      cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  const size_t smem = sizeof(float) * (size_t)width;
  if (!valid(j, width) || w == nullptr || smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  const bool vec = four_columns(j, width) && !odd(w) && !odd(out);
  auto kernel = vec ? depth_norm_kernel<T, 4> : depth_norm_kernel<T, 1>;
  if (int e = allow_smem(kernel, smem)) return e;
  return gllm_launch(kernel, dim3(n_rows), dim3(threads_for(width, vec ? 4 : 1)), smem, stream, j, rows, w, eps, out,
                     width);
}
}  // namespace

#define GLLM_DEPTH_EXPORTS(T, S)                                                                                       \
  GLLM_API int gllm_depth_conv_##S(const T* value, const float* parts, int n_parts, int64_t part_stride,               \
                                   const float* value_bias, const float* post_w, float post_eps, const float* resid,   \
                                   float* streams, int64_t stream_stride, int count, const float* depth_w,             \
                                   float* x_out, const float* conv_w, float* conv_state, const int* cu_q,              \
                                   const int* state_slots, T* out, int num_requests, int max_q_len, int width,         \
                                   int taps, cudaStream_t stream) {                                                    \
    const Joined<T> j{value, parts, n_parts, part_stride, value_bias, post_w, post_eps, resid, streams, stream_stride, \
                      count, depth_w};                                                                                 \
    return depth_conv_launch<T>(j, x_out, conv_w, conv_state, cu_q, state_slots, out, num_requests, max_q_len, width,  \
                                taps, stream);                                                                         \
  }                                                                                                                    \
  GLLM_API int gllm_depth_norm_##S(const T* value, const float* parts, int n_parts, int64_t part_stride,               \
                                   const float* value_bias, const float* post_w, float post_eps, const float* resid,   \
                                   float* streams, int64_t stream_stride, int count, const float* depth_w,             \
                                   const int* rows, int n_rows, const float* w, float eps, T* out, int width,          \
                                   cudaStream_t stream) {                                                              \
    const Joined<T> j{value, parts, n_parts, part_stride, value_bias, post_w, post_eps, resid, streams, stream_stride, \
                      count, depth_w};                                                                                 \
    return depth_norm_launch<T>(j, rows, n_rows, w, eps, out, width, stream);                                          \
  }

GLLM_DEPTH_EXPORTS(float, f32)
GLLM_DEPTH_EXPORTS(__nv_bfloat16, bf16)
