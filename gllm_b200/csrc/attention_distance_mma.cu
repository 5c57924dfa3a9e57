// Attention with a learned bias by distance of the bf16 path on the tensor cores, over the paged cache (see
// attention_distance.cu for the mechanism and the page layout).
//
// One CTA (4 warps) owns 64 rows = (64 / G') query tokens x G' query heads of one key head; key and value tiles of 64
// keys, aligned to absolute positions, are fetched page by page with cp.async in two stages; S = Q K^T and O += P V run
// as mma.sync m16n8k16 with fp32 accumulation, the softmax in base 2 with a running maximum and sum per row.  With a
// window only two stretches of tiles are visited: those of the first `keep_first` keys and those of the window.  Every
// tile's biases lie on (tokens of the tile + 63) distances per head: they are fetched into shared memory once per
// tile (a tile whose distances all lie past the table's end takes one value per head instead).  The sink is the
// start of the running maximum and sum.  DK and DV are the widths the tiles are built for; the heads may be narrower
// (multiples of 8): the rest is zero.  A CTA may take only a range of the visited tiles (`splits` > 1: single decoded
// tokens get enough CTAs to stream their keys); it then leaves (unnormalised O, maximum, sum) in fp32 and
// distance_merge combines the ranges.
#include "mma_utils.cuh"

namespace {
constexpr int BM = 64, BN = 64, THREADS = 128;
static_assert(THREADS == 2 * BN, "two threads fetch a key");
constexpr float LOG2E = 1.4426950408889634f;
constexpr float NEG_BIG = -1e30f;

template <int C>
__device__ __forceinline__ int swz(int row, int piece) {
  if (C % 8 == 0) return piece ^ (row & 7);
  return piece ^ ((row >> 1) & 3);
}

// bias: [hq][bias_len] and sink: [hq], both times log2(e).  partial: [split][token][head][dv] fp32, stats:
// [split][token][head][2] = (maximum in log2 units, sum).
template <int DK, int DV>
__global__ void __launch_bounds__(THREADS)
distance_mma_kernel(const __nv_bfloat16* __restrict__ q, int64_t q_stride, __nv_bfloat16* __restrict__ out,
                    int64_t out_stride, float* __restrict__ partial, float* __restrict__ stats, int n_tokens,
                    const __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_table, int bt_stride,
                    const int* __restrict__ cu_q, const int* __restrict__ ctx_lens, const int* __restrict__ slots,
                    const float* __restrict__ bias, int bias_len, const float* __restrict__ sink, int hq, int hkv, int gp,
                    int dk, int dv, int block_size, int num_pages, float scale_log2, int window, int keep_first,
                    int strip_ld, int splits, int tiles_per_split, int* __restrict__ status) {
  constexpr int CK = DK / 8, CV = DV / 8;
  constexpr int K_BYTES = BN * DK * 2, V_BYTES = BN * DV * 2;
  extern __shared__ __align__(128) unsigned char smem_raw[];
  unsigned char* q_sm = smem_raw;                       // [BM][DK]
  unsigned char* kv_sm = smem_raw + BM * DK * 2;        // [2 stages][K [BN][DK] | V [BN][DV]]
  float* strip = reinterpret_cast<float*>(kv_sm + 2 * (K_BYTES + V_BYTES));      // [gp][strip_ld]

  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.z;
  const int group = hq / hkv;
  const int tiles_per_kv = group / gp;
  const int kvh = blockIdx.y / tiles_per_kv;
  const int h0 = kvh * group + (blockIdx.y - kvh * tiles_per_kv) * gp;
  const int qt = BM / gp;
  const int tok_begin = cu_q[r], q_len = cu_q[r + 1] - tok_begin;
  const int n_qtiles = (q_len + qt - 1) / qt;
  const int split = blockIdx.x % splits;
  const int xt = blockIdx.x / splits;
  if (xt >= n_qtiles) return;
  const int qtile = n_qtiles - 1 - xt;                  // longest rows first
  const int t0 = qtile * qt;
  const int t_count = min(qt, q_len - t0);
  const int ctx = ctx_lens[r];
  const int* bt = block_table + (int64_t)slots[r] * bt_stride;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g8 = lane >> 2, t4 = lane & 3;

  const int pos_first = ctx + t0, pos_last = ctx + t0 + t_count - 1;
  // visited tiles: the first `kept`, then from tile `win` on
  const int wstart = window > 0 ? max(0, pos_first - window + 1) : 0;      // the first key any row's window holds
  int kept = window > 0 ? (keep_first + BN - 1) / BN : 0, win = wstart / BN;
  if (win <= kept) kept = win = 0;
  const int n_tiles = kept + pos_last / BN - win + 1;
  int it_first = 0, it_end = n_tiles;
  if (splits > 1) {
    it_first = split * tiles_per_split;
    it_end = min(n_tiles, it_first + tiles_per_split);
  }
  auto tile_of = [&](int it) { return it < kept ? it : win + it - kept; };

  const int64_t page_elems = (int64_t)hkv * block_size * (dk + dv);
  const int64_t v_region = (int64_t)hkv * block_size * dk;

  int qpos[2], row_tl[2], row_g[2];
  bool row_ok[2];
  float m_run[2], l_run[2], far_bias[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int rr = warp * 16 + g8 + 8 * i;
    row_tl[i] = rr / gp;
    row_g[i] = rr - row_tl[i] * gp;
    row_ok[i] = row_tl[i] < t_count;
    qpos[i] = pos_first + row_tl[i];
    m_run[i] = NEG_BIG;
    l_run[i] = 0.f;
    if (sink != nullptr && split == 0) {
      m_run[i] = sink[h0 + row_g[i]];
      l_run[i] = t4 == 0 ? 1.f : 0.f;                   // the row's four lanes are added at the end
    }
    far_bias[i] = bias[(int64_t)(h0 + row_g[i]) * bias_len + bias_len - 1];
  }
  float o[DV / 8][4];
#pragma unroll
  for (int nd = 0; nd < DV / 8; ++nd)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[nd][e] = 0.f;

  if (it_first < it_end) {
    for (int idx = threadIdx.x; idx < BM * CK; idx += THREADS) {
      const int rr = idx / CK, piece = idx - rr * CK;
      const int tl = rr / gp, g = rr - tl * gp;
      const bool ok = tl < t_count && piece * 8 < dk;
      const __nv_bfloat16* src = q + (int64_t)(tok_begin + t0 + tl) * q_stride + (int64_t)(h0 + g) * dk + piece * 8;
      cp_async16(smem_u32(q_sm + (rr * CK + swz<CK>(rr, piece)) * 16), ok ? src : q, ok);
    }
    // two threads a key: one page look-up each, then the key's 16-byte pieces in turn
    auto load_kv = [&](int tile, int stage) {
      unsigned char* k_dst = kv_sm + stage * (K_BYTES + V_BYTES);
      unsigned char* v_dst = k_dst + K_BYTES;
      const int row = threadIdx.x >> 1, half = threadIdx.x & 1;
      const int key = tile * BN + row;
      // (between the kept keys and the window a page may have been given back)
      bool ok = key <= pos_last && (key >= wstart || key < keep_first);
      int page = 0;
      if (ok) {
        page = bt[key / block_size];
        if (page < 0 || page >= num_pages) {
          atomicOr(status, GLLM_STATUS_PAGE_RANGE);
          ok = false;
          page = 0;
        }
      }
      const int off = key % block_size;
      const __nv_bfloat16* k_src = cache + (int64_t)page * page_elems + ((int64_t)kvh * block_size + off) * dk;
      const __nv_bfloat16* v_src = cache + (int64_t)page * page_elems + v_region + ((int64_t)kvh * block_size + off) * dv;
#pragma unroll
      for (int piece = half; piece < CK; piece += 2) {
        const bool take = ok && piece * 8 < dk;
        cp_async16(smem_u32(k_dst + (row * CK + swz<CK>(row, piece)) * 16), take ? k_src + piece * 8 : cache, take);
      }
#pragma unroll
      for (int piece = half; piece < CV; piece += 2) {
        const bool take = ok && piece * 8 < dv;
        cp_async16(smem_u32(v_dst + (row * CV + swz<CV>(row, piece)) * 16), take ? v_src + piece * 8 : cache, take);
      }
    };
    load_kv(tile_of(it_first), 0);
    cp_async_commit();
    uint32_t qf[DK / 16][4];

    for (int it = it_first; it < it_end; ++it) {
      const int stage = (it - it_first) & 1;
      const int kv0 = tile_of(it) * BN;
      if (it + 1 < it_end) {
        load_kv(tile_of(it + 1), stage ^ 1);
        cp_async_commit();
      }
      // the tile's biases: entry e of a head's strip is distance e + d_min (what lies ahead of a row is hidden below)
      const int d_min = pos_first - (kv0 + BN - 1);
      const bool far = d_min >= bias_len - 1;
      if (!far) {
        const int strip_n = qt + BN - 1;
        for (int g = 0; g < gp; ++g)
          for (int e = threadIdx.x; e < strip_n; e += THREADS)
            strip[g * strip_ld + e] = bias[(int64_t)(h0 + g) * bias_len + min(max(d_min + e, 0), bias_len - 1)];
      }
      if (it + 1 < it_end) cp_async_wait<1>();
      else cp_async_wait<0>();
      __syncthreads();
      if (it == it_first) {
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
          const int mat = lane >> 3, rl = lane & 7;
          const int row = warp * 16 + (mat & 1) * 8 + rl;
          const int piece = 2 * ks + (mat >> 1);
          ldmatrix_x4(qf[ks], smem_u32(q_sm + (row * CK + swz<CK>(row, piece)) * 16));
        }
      }
      const unsigned char* k_sm = kv_sm + stage * (K_BYTES + V_BYTES);
      const unsigned char* v_sm = k_sm + K_BYTES;

      float s[BN / 8][4];
#pragma unroll
      for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[nt][e] = 0.f;
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
#pragma unroll
        for (int np = 0; np < BN / 16; ++np) {
          const int mat = lane >> 3, rl = lane & 7;
          const int row = np * 16 + (mat >> 1) * 8 + rl;
          const int piece = 2 * ks + (mat & 1);
          uint32_t b[4];
          ldmatrix_x4(b, smem_u32(k_sm + (row * CK + swz<CK>(row, piece)) * 16));
          mma_bf16(s[2 * np], qf[ks], b[0], b[1]);
          mma_bf16(s[2 * np + 1], qf[ks], b[2], b[3]);
        }
      }
      // ---- scores with their biases in log2 units; hidden keys are marked
      const bool need_mask = (kv0 + BN - 1 > pos_first) || (t_count < qt) ||
                             (window > 0 && pos_last - kv0 >= window);
      float tmax[2] = {NEG_BIG, NEG_BIG};
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float* srow = strip + row_g[i] * strip_ld + row_tl[i] + BN - 1 - 2 * t4;
#pragma unroll
        for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const float b = far ? far_bias[i] : srow[-(nt * 8 + x)];
            float v = fmaf(s[nt][2 * i + x], scale_log2, b);
            if (need_mask) {
              const int key = kv0 + nt * 8 + 2 * t4 + x;
              if (!row_ok[i] || key > qpos[i] || (window > 0 && qpos[i] - key >= window && key >= keep_first)) v = NEG_BIG;
            }
            s[nt][2 * i + x] = v;
            tmax[i] = fmaxf(tmax[i], v);
          }
      }
      float corr[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 1));
        tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 2));
        const float m_new = fmaxf(m_run[i], tmax[i]);
        corr[i] = fast_exp2(m_run[i] - m_new);
        m_run[i] = m_new;
        l_run[i] *= corr[i];
      }
#pragma unroll
      for (int nt = 0; nt < BN / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = e >> 1;
          const float p = s[nt][e] <= NEG_BIG ? 0.f : fast_exp2(s[nt][e] - m_run[i]);
          s[nt][e] = p;
          l_run[i] += p;
        }
#pragma unroll
      for (int nd = 0; nd < DV / 8; ++nd) {
        o[nd][0] *= corr[0];
        o[nd][1] *= corr[0];
        o[nd][2] *= corr[1];
        o[nd][3] *= corr[1];
      }
      // ---- O += P V
#pragma unroll
      for (int kk = 0; kk < BN / 16; ++kk) {
        uint32_t a[4];
        a[0] = pack_bf16(s[2 * kk][0], s[2 * kk][1]);
        a[1] = pack_bf16(s[2 * kk][2], s[2 * kk][3]);
        a[2] = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
        a[3] = pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
#pragma unroll
        for (int nd2 = 0; nd2 < DV / 16; ++nd2) {
          const int mat = lane >> 3, rl = lane & 7;
          const int row = kk * 16 + (mat & 1) * 8 + rl;
          const int piece = 2 * nd2 + (mat >> 1);
          uint32_t b[4];
          ldmatrix_x4_trans(b, smem_u32(v_sm + (row * CV + swz<CV>(row, piece)) * 16));
          mma_bf16(o[2 * nd2], a, b[0], b[1]);
          mma_bf16(o[2 * nd2 + 1], a, b[2], b[3]);
        }
      }
      __syncthreads();
    }
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 1);
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 2);
    if (!row_ok[i]) continue;
    const int64_t token = tok_begin + t0 + row_tl[i];
    const int head = h0 + row_g[i];
    if (splits > 1) {
      const int64_t item = ((int64_t)split * n_tokens + token) * hq + head;
      float* dst = partial + item * dv;
#pragma unroll
      for (int nd = 0; nd < DV / 8; ++nd)
        if (nd * 8 < dv) *reinterpret_cast<float2*>(dst + nd * 8 + 2 * t4) = make_float2(o[nd][2 * i], o[nd][2 * i + 1]);
      if (t4 == 0) *reinterpret_cast<float2*>(stats + item * 2) = make_float2(m_run[i], l_run[i]);
    } else {
      const float mult = l_run[i] > 0.f ? 1.0f / l_run[i] : 0.f;
      __nv_bfloat16* dst = out + token * out_stride + (int64_t)head * dv;
#pragma unroll
      for (int nd = 0; nd < DV / 8; ++nd)
        if (nd * 8 < dv)
          *reinterpret_cast<__nv_bfloat162*>(dst + nd * 8 + 2 * t4) =
              __floats2bfloat162_rn(o[nd][2 * i] * mult, o[nd][2 * i + 1] * mult);
    }
  }
}

// ------------------------------------------------------------------ single tokens
// One CTA (4 warps) owns ONE token and up to 16 query heads of one key head (the rows of one mma tile); its warps take
// the visited key tiles (32 keys here) in turn, each with its own ring of cp.async stages and its own running maximum,
// sum and output, so that no warp waits for another until the end, where the four results are merged through shared
// memory.  A key's 16-byte pieces are fetched by neighbouring lanes.  With `splits` > 1 a CTA takes a range of the
// tiles and leaves its result for distance_merge.
constexpr int FN = 32, FW = 4;

template <int DK, int DV>
struct Few {
  static constexpr int K_BYTES = FN * DK * 2, V_BYTES = FN * DV * 2, STAGE = K_BYTES + V_BYTES;
  static constexpr int STAGES = DK + DV <= 128 ? 3 : 2;
  static constexpr int O_BYTES = FW * 16 * (DV + 4) * 4, ML_BYTES = 2 * FW * 16 * 4;
  static constexpr int RING = FW * STAGES * STAGE;
  static constexpr int SMEM = (RING > O_BYTES ? RING : O_BYTES) + ML_BYTES;
};

template <int DK, int DV>
__global__ void __launch_bounds__(FW * 32)
distance_few_kernel(const __nv_bfloat16* __restrict__ q, int64_t q_stride, __nv_bfloat16* __restrict__ out,
                    int64_t out_stride, float* __restrict__ partial, float* __restrict__ stats, int n_tokens,
                    const __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_table, int bt_stride,
                    const int* __restrict__ cu_q, const int* __restrict__ ctx_lens, const int* __restrict__ slots,
                    const float* __restrict__ bias, int bias_len, const float* __restrict__ sink, int hq, int hkv, int gp,
                    int dk, int dv, int block_size, int num_pages, float scale_log2, int window, int keep_first,
                    int splits, int tiles_per_split, int* __restrict__ status) {
  using S = Few<DK, DV>;
  constexpr int CK = DK / 8, CV = DV / 8;
  extern __shared__ __align__(128) unsigned char smem_raw[];
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g8 = lane >> 2, t4 = lane & 3;
  const int split = blockIdx.x, r = blockIdx.z;
  const int group = hq / hkv, tiles_per_kv = group / gp;
  const int kvh = blockIdx.y / tiles_per_kv;
  const int h0 = kvh * group + (blockIdx.y - kvh * tiles_per_kv) * gp;
  unsigned char* ring = smem_raw + warp * S::STAGES * S::STAGE;
  pdl_wait();
  const int64_t token = cu_q[r];
  const int pos = ctx_lens[r];
  const int* bt = block_table + (int64_t)slots[r] * bt_stride;

  const int wstart = window > 0 ? max(0, pos - window + 1) : 0;
  int kept = window > 0 ? (keep_first + FN - 1) / FN : 0, win = wstart / FN;
  if (win <= kept) kept = win = 0;
  const int n_tiles = kept + pos / FN - win + 1;
  const int it_end = splits > 1 ? min(n_tiles, (split + 1) * tiles_per_split) : n_tiles;
  const int it0 = (splits > 1 ? split * tiles_per_split : 0) + warp;
  auto tile_of = [&](int it) { return it < kept ? it : win + it - kept; };

  const int page_units = hkv * block_size * (dk + dv) / 8;      // in 16-byte units
  const int v_units = hkv * block_size * dk / 8;
  const uint4* pool = reinterpret_cast<const uint4*>(cache);
  auto load_tile = [&](int it, int stage) {
    const int key = tile_of(it) * FN + lane;
    int slot = -1, off = 0;                              // this lane's key: its page's and its own place
    if (key <= pos && (key >= wstart || key < keep_first)) {
      const int page = bt[key / block_size];
      if (page < 0 || page >= num_pages) atomicOr(status, GLLM_STATUS_PAGE_RANGE);
      else slot = page, off = key % block_size;
    }
    const int k_at = slot * page_units + (kvh * block_size + off) * (dk / 8);
    const int v_at = slot * page_units + v_units + (kvh * block_size + off) * (dv / 8);
    unsigned char* k_dst = ring + stage * S::STAGE;
    unsigned char* v_dst = k_dst + S::K_BYTES;
#pragma unroll
    for (int i = 0; i < CK; ++i) {
      const int idx = lane + 32 * i, row = idx / CK, piece = idx % CK;
      const int at = __shfl_sync(0xffffffffu, k_at, row);
      const bool take = __shfl_sync(0xffffffffu, slot, row) >= 0 && piece * 8 < dk;
      cp_async16(smem_u32(k_dst + (row * CK + swz<CK>(row, piece)) * 16), take ? pool + at + piece : pool, take);
    }
#pragma unroll
    for (int i = 0; i < CV; ++i) {
      const int idx = lane + 32 * i, row = idx / CV, piece = idx % CV;
      const int at = __shfl_sync(0xffffffffu, v_at, row);
      const bool take = __shfl_sync(0xffffffffu, slot, row) >= 0 && piece * 8 < dv;
      cp_async16(smem_u32(v_dst + (row * CV + swz<CV>(row, piece)) * 16), take ? pool + at + piece : pool, take);
    }
  };
  // the first tiles are on their way before the queries are read
#pragma unroll
  for (int s = 0; s + 1 < S::STAGES; ++s) {
    if (it0 + s * FW < it_end) load_tile(it0 + s * FW, s);
    cp_async_commit();
  }
  uint32_t qf[DK / 16][4];
  const __nv_bfloat16* q0 = q + token * q_stride + (int64_t)(h0 + min(g8, gp - 1)) * dk;
  const __nv_bfloat16* q1 = q + token * q_stride + (int64_t)(h0 + min(g8 + 8, gp - 1)) * dk;
#pragma unroll
  for (int ks = 0; ks < DK / 16; ++ks)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int c = ks * 16 + half * 8 + 2 * t4;
      const bool in = c < dk;
      qf[ks][2 * half] = in && g8 < gp ? *reinterpret_cast<const uint32_t*>(q0 + c) : 0u;
      qf[ks][2 * half + 1] = in && g8 + 8 < gp ? *reinterpret_cast<const uint32_t*>(q1 + c) : 0u;
    }
  const float* b0 = bias + (int64_t)(h0 + min(g8, gp - 1)) * bias_len;
  const float* b1 = bias + (int64_t)(h0 + min(g8 + 8, gp - 1)) * bias_len;
  const bool two = gp > 8;
  float m_run[2] = {NEG_BIG, NEG_BIG}, l_run[2] = {0.f, 0.f};
  float o[DV / 8][4];
#pragma unroll
  for (int nd = 0; nd < DV / 8; ++nd)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[nd][e] = 0.f;
  const int mat = lane >> 3, rl = lane & 7;

  int stage = 0;
  for (int it = it0; it < it_end; it += FW) {
    const int ahead = it + (S::STAGES - 1) * FW;
    if (ahead < it_end) load_tile(ahead, stage == 0 ? S::STAGES - 1 : stage - 1);
    cp_async_commit();
    const int kv0 = tile_of(it) * FN;
    float b[2][8];
#pragma unroll
    for (int nt = 0; nt < FN / 8; ++nt)
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int d = min(max(pos - (kv0 + nt * 8 + 2 * t4 + x), 0), bias_len - 1);
        b[0][2 * nt + x] = b0[d];
        b[1][2 * nt + x] = two ? b1[d] : 0.f;
      }
    cp_async_wait<S::STAGES - 1>();
    __syncwarp();
    const unsigned char* k_sm = ring + stage * S::STAGE;
    const unsigned char* v_sm = k_sm + S::K_BYTES;
    float s[FN / 8][4];
#pragma unroll
    for (int nt = 0; nt < FN / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nt][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks)
#pragma unroll
      for (int np = 0; np < FN / 16; ++np) {
        const int row = np * 16 + (mat >> 1) * 8 + rl, piece = 2 * ks + (mat & 1);
        uint32_t kb[4];
        ldmatrix_x4(kb, smem_u32(k_sm + (row * CK + swz<CK>(row, piece)) * 16));
        mma_bf16(s[2 * np], qf[ks], kb[0], kb[1]);
        mma_bf16(s[2 * np + 1], qf[ks], kb[2], kb[3]);
      }
    float tmax[2] = {NEG_BIG, NEG_BIG};
#pragma unroll
    for (int nt = 0; nt < FN / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = e >> 1, x = e & 1, key = kv0 + nt * 8 + 2 * t4 + x;
        const bool seen = key <= pos && (key >= wstart || key < keep_first);
        s[nt][e] = seen ? fmaf(s[nt][e], scale_log2, b[i][2 * nt + x]) : NEG_BIG;
        tmax[i] = fmaxf(tmax[i], s[nt][e]);
      }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 1));
      tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 2));
      const float m_new = fmaxf(m_run[i], tmax[i]);
      const float corr = fast_exp2(m_run[i] - m_new);
      m_run[i] = m_new;
      l_run[i] *= corr;
#pragma unroll
      for (int nd = 0; nd < DV / 8; ++nd) o[nd][2 * i] *= corr, o[nd][2 * i + 1] *= corr;
    }
#pragma unroll
    for (int nt = 0; nt < FN / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float p = s[nt][e] <= NEG_BIG ? 0.f : fast_exp2(s[nt][e] - m_run[e >> 1]);
        s[nt][e] = p;
        l_run[e >> 1] += p;
      }
#pragma unroll
    for (int kk = 0; kk < FN / 16; ++kk) {
      uint32_t a[4];
      a[0] = pack_bf16(s[2 * kk][0], s[2 * kk][1]);
      a[1] = pack_bf16(s[2 * kk][2], s[2 * kk][3]);
      a[2] = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
      a[3] = pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
#pragma unroll
      for (int nd2 = 0; nd2 < DV / 16; ++nd2) {
        const int row = kk * 16 + (mat & 1) * 8 + rl, piece = 2 * nd2 + (mat >> 1);
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, smem_u32(v_sm + (row * CV + swz<CV>(row, piece)) * 16));
        mma_bf16(o[2 * nd2], a, vb[0], vb[1]);
        mma_bf16(o[2 * nd2 + 1], a, vb[2], vb[3]);
      }
    }
    __syncwarp();                                        // the stage may be filled again
    stage = stage + 1 == S::STAGES ? 0 : stage + 1;
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- the four warps' results through shared memory
  float* o_sm = reinterpret_cast<float*>(smem_raw);      // [warp][16][DV + 4]
  float* ml = reinterpret_cast<float*>(smem_raw + S::SMEM - S::ML_BYTES);      // [warp][16] maxima, then sums
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 1);
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 2);
    const int row = g8 + 8 * i;
    if (t4 == 0) {
      ml[warp * 16 + row] = m_run[i];
      ml[(FW + warp) * 16 + row] = l_run[i];
    }
#pragma unroll
    for (int nd = 0; nd < DV / 8; ++nd)
      *reinterpret_cast<float2*>(o_sm + (warp * 16 + row) * (DV + 4) + nd * 8 + 2 * t4) =
          make_float2(o[nd][2 * i], o[nd][2 * i + 1]);
  }
  __syncthreads();
  const int row = threadIdx.x >> 3;
  if (row >= gp) return;
  const int head = h0 + row;
  float m = NEG_BIG, l = 0.f, w[FW];
  if (sink != nullptr && split == 0) m = sink[head], l = 1.f;
#pragma unroll
  for (int k = 0; k < FW; ++k) m = fmaxf(m, ml[k * 16 + row]);
  if (sink != nullptr && split == 0) l = fast_exp2(sink[head] - m);
#pragma unroll
  for (int k = 0; k < FW; ++k) {
    w[k] = ml[k * 16 + row] <= NEG_BIG ? 0.f : fast_exp2(ml[k * 16 + row] - m);
    l = fmaf(w[k], ml[(FW + k) * 16 + row], l);
  }
  const int64_t item = ((int64_t)split * n_tokens + token) * hq + head;
  const float mult = splits > 1 ? 1.f : (l > 0.f ? 1.0f / l : 0.f);
  for (int c = (threadIdx.x & 7) * 2; c < dv; c += 16) {
    float2 v = make_float2(0.f, 0.f);
#pragma unroll
    for (int k = 0; k < FW; ++k) {
      const float2 a = *reinterpret_cast<const float2*>(o_sm + (k * 16 + row) * (DV + 4) + c);
      v.x = fmaf(w[k], a.x, v.x);
      v.y = fmaf(w[k], a.y, v.y);
    }
    if (splits > 1)
      *reinterpret_cast<float2*>(partial + item * dv + c) = v;
    else
      *reinterpret_cast<__nv_bfloat162*>(out + token * out_stride + (int64_t)head * dv + c) =
          __floats2bfloat162_rn(v.x * mult, v.y * mult);
  }
  if (splits > 1 && (threadIdx.x & 7) == 0) *reinterpret_cast<float2*>(stats + item * 2) = make_float2(m, l);
}

// One warp per (token, head): the ranges' results, weighted by 2^(their maximum - the largest).
__global__ void __launch_bounds__(128)
distance_merge_kernel(const float* __restrict__ partial, const float* __restrict__ stats, __nv_bfloat16* __restrict__ out,
                      int64_t out_stride, int n_tokens, int hq, int dv, int splits) {
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t item = (int64_t)blockIdx.x * 4 + warp;
  const int64_t items = (int64_t)n_tokens * hq;
  if (item >= items) return;
  float2 mine = make_float2(NEG_BIG, 0.f);               // lane s: maximum and sum of range s (at most 32)
  if (lane < splits) mine = *reinterpret_cast<const float2*>(stats + ((int64_t)lane * items + item) * 2);
  const float big = warp_max(mine.y > 0.f ? mine.x : NEG_BIG);
  float w = mine.y > 0.f ? fast_exp2(mine.x - big) : 0.f;
  const float total = warp_sum(mine.y * w);
  w *= total > 0.f ? 1.0f / total : 0.f;
  float a[4] = {0.f, 0.f, 0.f, 0.f};                     // dv <= 128
#pragma unroll 8
  for (int s = 0; s < splits; ++s) {                     // ascending ranges: one order of the sums
    const float ws = __shfl_sync(0xffffffffu, w, s);
    const float* row = partial + ((int64_t)s * items + item) * dv;
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (lane + 32 * i < dv) a[i] = fmaf(row[lane + 32 * i], ws, a[i]);
  }
  const int64_t t = item / hq;
  __nv_bfloat16* dst = out + t * out_stride + (item - t * hq) * dv;
#pragma unroll
  for (int i = 0; i < 4; ++i)
    if (lane + 32 * i < dv) dst[lane + 32 * i] = __float2bfloat16_rn(a[i]);
}

inline int heads_per_tile(int group, int most) {        // the largest power of two that divides the group, at most `most`
  int gp = 1;
  while (gp < most && group % (2 * gp) == 0) gp *= 2;
  return gp;
}

template <int DK, int DV>
int distance_few_launch(const __nv_bfloat16* q, int64_t q_stride, __nv_bfloat16* out, int64_t out_stride, float* partial,
                        float* stats, int n_tokens, const __nv_bfloat16* cache, const int* block_table, int bt_stride,
                        const int* cu_q, const int* ctx_lens, const int* slots, const float* bias, int bias_len,
                        const float* sink, int num_requests, int hq, int hkv, int dk, int dv, int block_size,
                        int num_pages, float scale, int window, int keep_first, int splits, int tiles_per_split,
                        int* status, cudaStream_t stream) {
  const int group = hq / hkv, gp = heads_per_tile(group, 16);
  constexpr int smem = Few<DK, DV>::SMEM;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(distance_few_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
  }
  return gllm_launch(distance_few_kernel<DK, DV>, dim3(splits, hkv * (group / gp), num_requests), dim3(FW * 32), smem,
                     stream, q, q_stride, out, out_stride, partial, stats, n_tokens, cache, block_table, bt_stride, cu_q,
                     ctx_lens, slots, bias, bias_len, sink, hq, hkv, gp, dk, dv, block_size, num_pages, scale * LOG2E,
                     window, keep_first, splits, tiles_per_split, status);
}

template <int DK, int DV>
int distance_mma_launch(const __nv_bfloat16* q, int64_t q_stride, __nv_bfloat16* out, int64_t out_stride, float* partial,
                        float* stats, int n_tokens, const __nv_bfloat16* cache, const int* block_table, int bt_stride,
                        const int* cu_q, const int* ctx_lens, const int* slots, const float* bias, int bias_len,
                        const float* sink, int num_requests, int max_q_len, int hq, int hkv, int dk, int dv,
                        int block_size, int num_pages, float scale, int window, int keep_first, int splits,
                        int tiles_per_split, int* status, cudaStream_t stream) {
  const int group = hq / hkv, gp = heads_per_tile(group, BM), qt = BM / gp;
  // a strip's start is 8 banks after the one before it, so that the heads of a warp's rows read different banks
  const int strip_ld = (qt + BN - 1 + 23) / 32 * 32 + 8;
  const size_t smem = (size_t)BM * DK * 2 + 2 * (size_t)BN * (DK + DV) * 2 + sizeof(float) * (size_t)gp * strip_ld;
  if (smem > 48 * 1024) {
    cudaError_t e =
        cudaFuncSetAttribute(distance_mma_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  dim3 grid(((max_q_len + qt - 1) / qt) * splits, hkv * (group / gp), num_requests);
  return gllm_launch(distance_mma_kernel<DK, DV>, grid, dim3(THREADS), smem, stream, q, q_stride, out, out_stride, partial,
                     stats, n_tokens, cache, block_table, bt_stride, cu_q, ctx_lens, slots, bias, bias_len, sink, hq, hkv,
                     gp, dk, dv, block_size, num_pages, scale * LOG2E, window, keep_first, strip_ld, splits,
                     tiles_per_split, status);
}
}  // namespace

// Query tokens and keys per tile of a launch (the caller sizes its split decision with them).
GLLM_API int gllm_attention_distance_mma_tokens_per_tile(int hq, int hkv) { return BM / heads_per_tile(hq / hkv, BM); }
// CTAs per request and range of the kernel for single tokens.
GLLM_API int gllm_attention_distance_few_tiles(int hq, int hkv) { return hq / heads_per_tile(hq / hkv, 16); }

// `single`: every one of these requests brings one token (requests r of cu_q, ctx_lens, slots); tiles_per_split then counts
// tiles of 32 keys.  bias, sink: times log2(e).  partial: fp32 [splits][n_tokens][hq][dv]; stats: fp32 [splits][n_tokens][hq][2] (scratch,
// with splits > 1 only).
GLLM_API int gllm_attention_distance_mma(const __nv_bfloat16* q, int64_t q_stride, __nv_bfloat16* out, int64_t out_stride,
                                         float* partial, float* stats, int n_tokens, const __nv_bfloat16* cache,
                                         const int* block_table, int bt_stride, const int* cu_q, const int* ctx_lens,
                                         const int* slots, const float* bias, int bias_len, const float* sink,
                                         int num_requests, int max_q_len, int hq, int hkv, int dk, int dv, int block_size,
                                         int num_pages, float scale, int window, int keep_first, int single, int splits,
                                         int tiles_per_split, int* status, cudaStream_t stream) {
  if (num_requests <= 0 || max_q_len <= 0 || n_tokens <= 0) return 0;
  if (hq <= 0 || hkv <= 0 || hq % hkv || num_requests > 65535 || (q_stride % 8) || (out_stride % 2) || dk < 8 || dv < 8 ||
      (dk % 8) || (dv % 8) || dk > 128 || dv > 128 || bias == nullptr || bias_len < 1 || window < 0 || keep_first < 0 ||
      splits < 1 || splits > 32 || (splits > 1 && (tiles_per_split < 1 || partial == nullptr || stats == nullptr)) ||
      (reinterpret_cast<uintptr_t>(q) & 15) || (reinterpret_cast<uintptr_t>(cache) & 15) ||
      (reinterpret_cast<uintptr_t>(out) & 3) ||
      (single && (int64_t)num_pages * hkv * block_size * (dk + dv) / 8 > 0x7fffffffLL))
    return (int)cudaErrorInvalidValue;
  auto built = [](int d) { return d <= 32 ? 32 : (d <= 64 ? 64 : 128); };
  const int bk = built(dk), bv = built(dv);
  int rc = (int)cudaErrorInvalidValue;
#define GLLM_DIST(A, B)                                                                                                \
  if (bk == A && bv == B && single)                                                                                    \
    rc = distance_few_launch<A, B>(q, q_stride, out, out_stride, partial, stats, n_tokens, cache, block_table, bt_stride, \
                                   cu_q, ctx_lens, slots, bias, bias_len, sink, num_requests, hq, hkv, dk, dv,         \
                                   block_size, num_pages, scale, window, keep_first, splits, tiles_per_split, status,  \
                                   stream);                                                                            \
  if (bk == A && bv == B && !single)                                                                                   \
    rc = distance_mma_launch<A, B>(q, q_stride, out, out_stride, partial, stats, n_tokens, cache, block_table, bt_stride, \
                                   cu_q, ctx_lens, slots, bias, bias_len, sink, num_requests, max_q_len, hq, hkv, dk,  \
                                   dv, block_size, num_pages, scale, window, keep_first, splits, tiles_per_split,      \
                                   status, stream);
  GLLM_DIST(32, 32) GLLM_DIST(32, 64) GLLM_DIST(32, 128)
  GLLM_DIST(64, 32) GLLM_DIST(64, 64) GLLM_DIST(64, 128)
  GLLM_DIST(128, 32) GLLM_DIST(128, 64) GLLM_DIST(128, 128)
#undef GLLM_DIST
  if (rc != 0 || splits == 1) return rc;
  const int64_t blocks = ((int64_t)n_tokens * hq + 3) / 4;
  if (blocks > 0x7fffffffLL) return (int)cudaErrorInvalidValue;
  return gllm_launch(distance_merge_kernel, dim3((unsigned)blocks), dim3(128), 0, stream, (const float*)partial,
                     (const float*)stats, out, out_stride, n_tokens, hq, dv, splits);
}
