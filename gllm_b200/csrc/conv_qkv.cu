// From one attention layer's fused projection [q heads | k heads | v heads] to rotated queries and stored keys and
// values, for layers whose projections pass a short causal convolution over time before anything else:
//   u_t    = projection (rounded to T, as the product rounds it) + bias
//   y_t    = sum_j w[j] * u_(t - taps + 1 + j), one filter per channel; inputs before the request's first token are 0
//   q, k   : y / sqrt(mean(y^2) + eps) * norm weight, per head; then the neighbours (2i, 2i+1) of the first rotary_dim
//            columns turn by position * inv_freq[i], sine and cosine times `magnitude`
//   v      : y
// q goes to q_out [n, hq * dp], k and v into the token's cache slot, layout [page][k|v][kv_head][block_size][dp]; a head's
// columns behind its width are written as zeros.  A layer that attends over another's keys has q heads alone
// (own_kv = 0).  Everything between the projection and the one rounding to T at the end is fp32.
//
// The last taps - 1 inputs u of every request are its state [slots, taps - 1, channels] (fp32), so a prompt may be cut
// anywhere.  A warp takes `32 / lanes` heads over a run of neighbouring tokens of one request, eight columns a lane: the
// convolution's window stays in registers and neighbouring tokens of a run go through the norm and the rotation together.  The sines and cosines of
// the run's positions are computed once per block, into shared memory.  The warp that opens a
// portion is the only reader of its heads' state (runs are at least taps - 1 tokens long) and also writes the new one,
// after the reads.  The projection may arrive as unsummed fp32 splits (summed in ascending order).
#include "common.cuh"

#include <algorithm>

namespace {
constexpr int CQ_COLS = 8;            // columns of a head per lane
constexpr int CQ_WARPS = 4;
// tokens taken side by side, blocks an SM (of the kernels for short filters)
#ifndef GLLM_CONV_QKV_AHEAD
#define GLLM_CONV_QKV_AHEAD 2
#endif
#ifndef GLLM_CONV_QKV_BLOCKS
#define GLLM_CONV_QKV_BLOCKS 4
#endif
constexpr int CQ_AHEAD = GLLM_CONV_QKV_AHEAD;
constexpr int CQ_MAX_TAPS = 16;

template <typename T> struct alignas(16) Row8 {
  T v[CQ_COLS];
};

__device__ __forceinline__ void load16(Row8<__nv_bfloat16>& r, const __nv_bfloat16* p) {
  *reinterpret_cast<uint4*>(r.v) = *reinterpret_cast<const uint4*>(p);
}
__device__ __forceinline__ void load16(Row8<float>& r, const float* p) {
  reinterpret_cast<float4*>(r.v)[0] = reinterpret_cast<const float4*>(p)[0];
  reinterpret_cast<float4*>(r.v)[1] = reinterpret_cast<const float4*>(p)[1];
}
__device__ __forceinline__ void store16(__nv_bfloat16* p, const Row8<__nv_bfloat16>& r) {
  *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(r.v);
}
__device__ __forceinline__ void store16(float* p, const Row8<float>& r) {
  reinterpret_cast<float4*>(p)[0] = reinterpret_cast<const float4*>(r.v)[0];
  reinterpret_cast<float4*>(p)[1] = reinterpret_cast<const float4*>(r.v)[1];
}
// eight fp32 values, `nc` of them real (VEC: all eight or none, and the address is 16-byte aligned)
template <bool VEC> __device__ __forceinline__ void load_f8(const float* p, int nc, float (&v)[CQ_COLS]) {
  if (VEC) {
    if (nc > 0) {
      const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
      v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
      return;
    }
#pragma unroll
    for (int e = 0; e < CQ_COLS; ++e) v[e] = 0.f;
  } else {
#pragma unroll
    for (int e = 0; e < CQ_COLS; ++e) v[e] = e < nc ? p[e] : 0.f;
  }
}
template <bool VEC> __device__ __forceinline__ void store_f8(float* p, int nc, const float (&v)[CQ_COLS]) {
  if (VEC) {
    if (nc > 0) {
      reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
      reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
    }
  } else {
#pragma unroll
    for (int e = 0; e < CQ_COLS; ++e)
      if (e < nc) p[e] = v[e];
  }
}

template <typename T> struct ConvQkv {
  const T* proj;                // [n, channels] at `stride`, or null: parts
  int64_t stride;
  const float* parts;           // [n_parts][n, channels]
  int n_parts;
  int64_t part_stride;
  const float* bias;            // [channels] or null
  const float* conv_w;          // [taps][channels], last row: the current token
  float* conv_state;            // [slots][taps - 1][channels]
  const int *cu_q, *state_slots, *positions;
  const float *q_norm, *k_norm; // [dk]
  float eps;
  const float* inv_freq;        // [rotary_dim / 2] or null
  int rotary_dim;
  float magnitude;
  const int* slot_mapping;
  T *q_out, *cache;
  int hq, hkv, own_kv, dk, dv, dp, taps, block_size, num_pages;
  int* status;
};

// grid (runs, requests, groups of CQ_WARPS * 32 / lanes heads).  TM: the most taps (a filter of fewer is padded with
// zeros in front).  VEC: head widths and row starts are multiples of 8 elements.  Shared memory: the norm weights
// [q | k][lanes * 8], the turns of the run's tokens [run][pairs of the rotation, padded to 4] (cosine, sine), and the
// tokens' cache rows [run].
template <typename T, int TM, bool VEC>
__global__ void __launch_bounds__(CQ_WARPS * 32, TM <= 4 ? GLLM_CONV_QKV_BLOCKS : 1)
conv_qkv_kernel(const ConvQkv<T> a, int run, int lanes) {
  extern __shared__ __align__(16) float cq_smem[];
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane & (lanes - 1);
  const int heads = a.hq + (a.own_kv ? 2 * a.hkv : 0);
  const int unit = ((int)blockIdx.z * CQ_WARPS + warp) * (32 / lanes) + lane / lanes;
  const int q_cols = a.hq * a.dk, k_cols = a.hkv * a.dk;
  const int channels = q_cols + (a.own_kv ? k_cols + a.hkv * a.dv : 0);
  const bool is_q = unit < a.hq, is_qk = unit < a.hq + a.hkv, live = unit < heads;
  const int d = is_qk ? a.dk : a.dv, c0 = sub * CQ_COLS;
  const int head0 = is_q ? unit * a.dk : is_qk ? q_cols + (unit - a.hq) * a.dk : q_cols + k_cols + (unit - a.hq - a.hkv) * a.dv;
  const int ch = head0 + c0;
  const int nc = live ? min(max(d - c0, 0), CQ_COLS) : 0;    // real columns of this lane
  const int keep = a.taps - 1;
  const int pairs = a.inv_freq ? a.rotary_dim / 2 : 0, pairs4 = (pairs + 3) & ~3;
  const bool turns = is_qk && c0 < 2 * pairs;
  const int padded = lanes * CQ_COLS;
  float* norm_s = cq_smem;
  float2* turn = reinterpret_cast<float2*>(cq_smem + 2 * padded);
  int* where = reinterpret_cast<int*>(turn + run * pairs4);

  // what is older than the step: the filters, the bias, the norm weights
  float wt[TM][CQ_COLS], bias[CQ_COLS];
#pragma unroll
  for (int k = 0; k < TM; ++k) {
    const int tap = k - (TM - a.taps);
    load_f8<VEC>(a.conv_w + (int64_t)max(tap, 0) * channels + ch, tap >= 0 ? nc : 0, wt[k]);
  }
  load_f8<VEC>(a.bias + ch, a.bias ? nc : 0, bias);
  for (int c = threadIdx.x; c < padded; c += CQ_WARPS * 32) {
    norm_s[c] = c < a.dk ? a.q_norm[c] : 0.f;
    norm_s[padded + c] = c < a.dk && a.own_kv ? a.k_norm[c] : 0.f;
  }
  const float* nw = norm_s + (is_q ? 0 : padded) + c0;

  pdl_wait();
  const int r = blockIdx.y;
  const int t0 = a.cu_q[r], len = a.cu_q[r + 1] - t0;
  const int begin = blockIdx.x * run;
  if (begin >= len) return;                                  // the whole block together
  const int end = min(begin + run, len);
  // (columns behind the rotated ones turn by nothing)
  for (int idx = threadIdx.x; idx < (end - begin) * pairs4; idx += CQ_WARPS * 32) {
    const int t = idx / pairs4, i = idx - t * pairs4;
    float s = 0.f, c = 1.f;
    if (i < pairs) {
      sincosf((float)a.positions[t0 + begin + t] * a.inv_freq[i], &s, &c);
      s *= a.magnitude;
      c *= a.magnitude;
    }
    turn[idx] = make_float2(c, s);
  }
  // a token's first row of the cache, in rows of dp elements (head h of keys and values: h * block_size rows on)
  for (int t = threadIdx.x; t < end - begin; t += CQ_WARPS * 32) {
    int row = -1;
    const int slot = a.slot_mapping ? a.slot_mapping[t0 + begin + t] : -1;
    if (slot >= 0) {
      const int page = slot / a.block_size;
      if (page >= a.num_pages) atomicOr(a.status, GLLM_STATUS_PAGE_RANGE);
      else row = page * 2 * a.hkv * a.block_size + (slot - page * a.block_size);
    }
    where[t] = row;
  }
  __syncthreads();

  // row i of the request's portion as the product left it (rounded to T)
  auto fetch = [&](int i, Row8<T>& out) {
    const int64_t n = t0 + i;
    if (a.parts) {
      float s[CQ_COLS];
#pragma unroll
      for (int e = 0; e < CQ_COLS; ++e) s[e] = 0.f;
      const float* p = a.parts + n * channels + ch;
      for (int k = 0; k < a.n_parts; k += 4) {
        float v[4][CQ_COLS];
#pragma unroll
        for (int q = 0; q < 4; ++q) load_f8<VEC>(p + (int64_t)(k + q) * a.part_stride, k + q < a.n_parts ? nc : 0, v[q]);
#pragma unroll
        for (int q = 0; q < 4; ++q)
#pragma unroll
          for (int e = 0; e < CQ_COLS; ++e) s[e] += v[q][e];
      }
#pragma unroll
      for (int e = 0; e < CQ_COLS; ++e) out.v[e] = from_float<T>(s[e]);
    } else if (VEC) {
      if (nc > 0) {
        load16(out, a.proj + n * a.stride + ch);
      } else {
#pragma unroll
        for (int e = 0; e < CQ_COLS; ++e) out.v[e] = from_float<T>(0.f);
      }
    } else {
#pragma unroll
      for (int e = 0; e < CQ_COLS; ++e) out.v[e] = e < nc ? a.proj[n * a.stride + ch + e] : from_float<T>(0.f);
    }
  };
  auto input = [&](const Row8<T>& raw, float (&u)[CQ_COLS]) {
#pragma unroll
    for (int e = 0; e < CQ_COLS; ++e) u[e] = to_float(raw.v[e]) + bias[e];   // (0 where the lane has no column)
  };

  // the window before the run's first token, right-aligned: win[TM - 2] is the token before it
  float win[TM][CQ_COLS];
  float* cs = keep > 0 ? a.conv_state + (int64_t)a.state_slots[r] * keep * channels + ch : nullptr;
#pragma unroll
  for (int k = 0; k < TM - 1; ++k) {
    const int back = TM - 1 - k;                             // so many tokens before the run's first
#pragma unroll
    for (int e = 0; e < CQ_COLS; ++e) win[k][e] = 0.f;
    if (back <= keep) {
      if (begin == 0) {
        load_f8<VEC>(cs + (int64_t)(keep - back) * channels, nc, win[k]);
      } else {
        Row8<T> raw;
        fetch(begin - back, raw);
        input(raw, win[k]);
      }
    }
  }

  auto convolve = [&](const Row8<T>& raw, float (&y)[CQ_COLS]) {
    input(raw, win[TM - 1]);
#pragma unroll
    for (int e = 0; e < CQ_COLS; ++e) {
      y[e] = 0.f;
#pragma unroll
      for (int k = 0; k < TM; ++k) y[e] = fmaf(wt[k][e], win[k][e], y[e]);
    }
#pragma unroll
    for (int k = 0; k + 1 < TM; ++k)
#pragma unroll
      for (int e = 0; e < CQ_COLS; ++e) win[k][e] = win[k + 1][e];
  };
  auto norm_and_turn = [&](float (&y)[CQ_COLS], float ss, int t) {
    if (!is_qk) return;
    const float inv = rsqrtf(ss / (float)a.dk + a.eps);
#pragma unroll
    for (int e = 0; e < CQ_COLS; e += 4) {
      const float4 w = *reinterpret_cast<const float4*>(nw + e);
      y[e] *= inv * w.x, y[e + 1] *= inv * w.y, y[e + 2] *= inv * w.z, y[e + 3] *= inv * w.w;
    }
    if (!turns) return;
#pragma unroll
    for (int i = 0; i < CQ_COLS / 2; i += 2) {               // two pairs: cosine, sine, cosine, sine
      const float4 c = *reinterpret_cast<const float4*>(turn + (t - begin) * pairs4 + c0 / 2 + i);
      const float u0 = y[2 * i], v0 = y[2 * i + 1], u1 = y[2 * i + 2], v1 = y[2 * i + 3];
      y[2 * i] = u0 * c.x - v0 * c.y;
      y[2 * i + 1] = v0 * c.x + u0 * c.y;
      y[2 * i + 2] = u1 * c.z - v1 * c.w;
      y[2 * i + 3] = v1 * c.z + u1 * c.w;
    }
  };
  auto put = [&](const float (&y)[CQ_COLS], int t) {
    T* dst = nullptr;
    if (is_q) dst = a.q_out + ((int64_t)(t0 + t) * a.hq + unit) * a.dp;
    else if (live && where[t - begin] >= 0) dst = a.cache + ((int64_t)where[t - begin] + (unit - a.hq) * a.block_size) * a.dp;
    if (dst && c0 < a.dp) {
      Row8<T> o;
#pragma unroll
      for (int e = 0; e < CQ_COLS; ++e) o.v[e] = from_float<T>(VEC || e < nc ? y[e] : 0.f);
      store16(dst + c0, o);
    }
  };
  auto head_sum = [&](float ss) {
    for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    return ss;
  };
  auto squares = [](const float (&y)[CQ_COLS]) {
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < CQ_COLS; ++e) ss = fmaf(y[e], y[e], ss);
    return ss;
  };

  int t = begin;
  for (; t + CQ_AHEAD <= end; t += CQ_AHEAD) {               // CQ_AHEAD tokens side by side
    Row8<T> raw[CQ_AHEAD];
    float y[CQ_AHEAD][CQ_COLS], ss[CQ_AHEAD];
#pragma unroll
    for (int q = 0; q < CQ_AHEAD; ++q) fetch(t + q, raw[q]);
#pragma unroll
    for (int q = 0; q < CQ_AHEAD; ++q) convolve(raw[q], y[q]), ss[q] = squares(y[q]);
    for (int o = lanes >> 1; o > 0; o >>= 1)
#pragma unroll
      for (int q = 0; q < CQ_AHEAD; ++q) ss[q] += __shfl_xor_sync(0xffffffffu, ss[q], o);
#pragma unroll
    for (int q = 0; q < CQ_AHEAD; ++q) norm_and_turn(y[q], ss[q], t + q);
#pragma unroll
    for (int q = 0; q < CQ_AHEAD; ++q) put(y[q], t + q);
  }
#pragma unroll 1
  for (; t < end; ++t) {
    Row8<T> raw;
    float y[CQ_COLS];
    fetch(t, raw);
    convolve(raw, y);
    norm_and_turn(y, head_sum(squares(y)), t);
    put(y, t);
  }

  // the request's new state: its last taps - 1 inputs
  if (begin == 0 && keep > 0) {
    if (end == len) {                                        // one run holds the portion: the window has them
#pragma unroll
      for (int k = 0; k < TM - 1; ++k) {
        const int idx = k - (TM - 1 - keep);
        if (idx >= 0) store_f8<VEC>(cs + (int64_t)idx * channels, nc, win[k]);
      }
    } else {                                                 // (len > run >= keep: all of them are rows of this portion)
      for (int idx = 0; idx < keep; ++idx) {
        Row8<T> raw;
        float u[CQ_COLS];
        fetch(len - keep + idx, raw);
        input(raw, u);
        store_f8<VEC>(cs + (int64_t)idx * channels, nc, u);
      }
    }
  }
}

template <typename T>
int conv_qkv_launch(const ConvQkv<T>& a, int num_requests, int max_q_len, cudaStream_t stream) {
  if (num_requests <= 0 || max_q_len <= 0) return 0;
  const int widest = a.dk > a.dv ? a.dk : a.dv;
  if (a.taps < 1 || a.taps > CQ_MAX_TAPS || a.dp % CQ_COLS || a.dp < widest || a.dp > 256 || a.rotary_dim < 0 ||
      a.rotary_dim > a.dk || (a.rotary_dim & 1) || num_requests > 65535 || a.hq < 1 || a.hkv < 1 || a.n_parts > 16 ||
      (reinterpret_cast<uintptr_t>(a.q_out) & 15) || (reinterpret_cast<uintptr_t>(a.cache) & 15) ||
      (a.taps > 1 && a.conv_state == nullptr) || (a.slot_mapping != nullptr && a.cache == nullptr) ||
      (int64_t)a.num_pages * 2 * a.hkv * a.block_size > 0x7fffffff)
    return (int)cudaErrorInvalidValue;
  int lanes = 1;
  while (lanes * CQ_COLS < a.dp) lanes *= 2;
  const int heads = a.hq + (a.own_kv ? 2 * a.hkv : 0), per_block = CQ_WARPS * (32 / lanes);
  const int groups = (heads + per_block - 1) / per_block;
  // Runs as short as all blocks still fit the machine at once (their turns fit 40 KB of shared memory), never shorter
  // than the state.
  const int keep = a.taps - 1, pairs4 = a.inv_freq ? (a.rotary_dim / 2 + 3) & ~3 : 0;
  const int64_t places = (int64_t)gllm_sm_count() * GLLM_CONV_QKV_BLOCKS / ((int64_t)num_requests * groups);
  int run = (int)((max_q_len + (places > 1 ? places : 1) - 1) / (places > 1 ? places : 1));
  run = std::min((std::max(run, 4) + 1) & ~1, std::min(256, 40 * 1024 / (8 * pairs4 + 4)));
  if (run < keep) run = keep;
  auto misaligned = [](const void* p) { return p != nullptr && (reinterpret_cast<uintptr_t>(p) & 15) != 0; };
  const bool vec = a.dk % CQ_COLS == 0 && a.dv % CQ_COLS == 0 && (a.proj == nullptr || a.stride % CQ_COLS == 0) &&
                   a.part_stride % 4 == 0 && !misaligned(a.proj) && !misaligned(a.parts) && !misaligned(a.bias) &&
                   !misaligned(a.conv_w) && !misaligned(a.conv_state) && !misaligned(a.q_norm) && !misaligned(a.k_norm);
  const size_t smem = sizeof(float) * 2 * lanes * CQ_COLS + sizeof(int) * (size_t)run + sizeof(float2) * (size_t)run * pairs4;
  const dim3 grid((max_q_len + run - 1) / run, num_requests, groups);
#define GLLM_CONV_QKV(TM)                                                                                             \
  return vec ? gllm_launch(conv_qkv_kernel<T, TM, true>, grid, dim3(CQ_WARPS * 32), smem, stream, a, run, lanes)        \
             : gllm_launch(conv_qkv_kernel<T, TM, false>, grid, dim3(CQ_WARPS * 32), smem, stream, a, run, lanes)
  if (a.taps <= 2) GLLM_CONV_QKV(2);
  if (a.taps <= 4) GLLM_CONV_QKV(4);
  if (a.taps <= 8) GLLM_CONV_QKV(8);
  GLLM_CONV_QKV(16);
#undef GLLM_CONV_QKV
}
}  // namespace

#define GLLM_CONV_QKV_EXPORT(T, S)                                                                                     \
  GLLM_API int gllm_conv_qkv_##S(const T* proj, int64_t stride, const float* parts, int n_parts, int64_t part_stride,  \
                                 const float* bias, const float* conv_w, float* conv_state, const int* cu_q,           \
                                 const int* state_slots, const int* positions, const float* q_norm,                    \
                                 const float* k_norm, float eps, const float* inv_freq, int rotary_dim,                \
                                 float magnitude, const int* slot_mapping, T* q_out, T* cache, int num_requests,       \
                                 int max_q_len, int hq, int hkv, int own_kv, int dk, int dv, int dp, int taps,         \
                                 int block_size, int num_pages, int* status, cudaStream_t stream) {                    \
    const ConvQkv<T> a{proj, stride, parts, n_parts, part_stride, bias, conv_w, conv_state, cu_q, state_slots,         \
                       positions, q_norm, k_norm, eps, inv_freq, rotary_dim, magnitude, slot_mapping, q_out, cache,    \
                       hq, hkv, own_kv, dk, dv, dp, taps, block_size, num_pages, status};                              \
    return conv_qkv_launch<T>(a, num_requests, max_q_len, stream);                                                     \
  }

GLLM_CONV_QKV_EXPORT(float, f32)
GLLM_CONV_QKV_EXPORT(__nv_bfloat16, bf16)
