// Differential attention: every head is two maps over one value head, each an ordinary causal softmax attention with
// queries and keys of its own; the head's output is the first map's minus a share of the second's, divided by its root
// mean square.  Grouped key heads.  The cache holds one row [key 1 | key 2 | value] per position and key head.
//
//   differential_prep     per token and head: the projections pass a short causal convolution over time (channel by
//                         channel, the sequence's last taps - 1 inputs are state), queries and keys are divided by their
//                         root mean square per map (times a weight that all heads and maps share) and turned by the
//                         token's position, channel 2i with 2i + 1; queries go to `q_out`, keys and values into the
//                         token's row of the layer's pages.
//   two_map_attention     both maps of a token's heads over the pages, 32-bit multiply-adds: decode steps, short runs, 32-bit
//                         models, head sizes the tensor-core form (attention_prefill_tcgen05.cu) does not take.  Leaves the
//                         maps' results, or their parts when the keys are split over blocks.
//   differential_combine  joins the parts, o = a1 - share * a2, o / sqrt(mean(o^2) + eps) * gain.
#include "common.cuh"

namespace bt {

constexpr int DA_MAX_TAPS = 16;
constexpr int DA_TK = 32;          // keys a tile: one per lane
constexpr int DA_MAX_SPLITS = 64;

struct DiffPrepArgs {
  const void* proj;                // rows [q | k | v]: 2 heads dim, 2 kv_heads dim, kv_heads vdim channels
  long long row_stride;
  const float* conv;               // [taps][channels]
  float* state;                    // [slots][taps - 1][channels], the newest input last
  const int *slots, *seq_start, *token_seq, *positions, *table;
  const float *q_weight, *k_weight, *inv_freq;
  float eps, rot_size;             // rot_size multiplies sine and cosine
  int rot_dims, taps, table_stride, table_len, page_size;
  void* pool;                      // [pages][kv_heads][page_size][2 dim + vdim]
  void* q_out;                     // rows of 2 heads q_pad channels
  int n_tokens, n_heads, n_kv_heads, dim, vdim, q_pad;
  int shift_state;                 // every sequence brings one token: the kernel moves the state on itself
  int pairs_ok;                    // two adjacent channels may be read and written as one word
};

template <typename T>
__device__ __forceinline__ float2 da_pair(const T* p, bool second, bool word);
template <>
__device__ __forceinline__ float2 da_pair<float>(const float* p, bool second, bool word) {
  if (word && second) return *reinterpret_cast<const float2*>(p);
  return make_float2(p[0], second ? p[1] : 0.f);
}
template <>
__device__ __forceinline__ float2 da_pair<__nv_bfloat16>(const __nv_bfloat16* p, bool second, bool word) {
  if (word && second) return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
  return make_float2(to_float(p[0]), second ? to_float(p[1]) : 0.f);
}

__device__ __forceinline__ void da_store_pair(float* p, float a, float b, bool second, bool word) {
  if (word && second) { *reinterpret_cast<float2*>(p) = make_float2(a, b); return; }
  p[0] = a;
  if (second) p[1] = b;
}
__device__ __forceinline__ void da_store_pair(__nv_bfloat16* p, float a, float b, bool second, bool word) {
  if (word && second) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); return; }
  p[0] = __float2bfloat16_rn(a);
  if (second) p[1] = __float2bfloat16_rn(b);
}

constexpr int DA_PREP_WARPS = 8;

// A warp takes one unit (a map of a query or key head, or 64 PJ channels of a value head) of RUN consecutive tokens; a lane
// owns PJ channel pairs of it, 64 channels apart.  The run's inputs are asked for together; where TAPS says how many taps
// there are (0: any number), taps and the inputs before the run stay in registers too, so every input is read once a run.
// The block's warps take the same tokens: sines and cosines of the run are formed once for all of them.
template <typename T, int TAPS, int PJ, int RUN>
__global__ void __launch_bounds__(DA_PREP_WARPS * 32) differential_prep_kernel(DiffPrepArgs p) {
  extern __shared__ float2 turn[];       // [RUN][rot_dims / 2]: (cosine, sine) times rot_size
  const int lane = threadIdx.x & 31;
  const int v_pieces = (p.vdim + 64 * PJ - 1) / (64 * PJ);
  const int q_units = 2 * p.n_heads, k_units = 2 * p.n_kv_heads, units = q_units + k_units + p.n_kv_heads * v_pieces;
  const int unit = blockIdx.y * DA_PREP_WARPS + (threadIdx.x >> 5);
  const int taps = TAPS > 0 ? TAPS : p.taps;
  const int channels = (q_units + k_units) * p.dim + p.n_kv_heads * p.vdim;
  const bool works = unit < units, is_q = unit < q_units, is_k = !is_q && unit < q_units + k_units;
  const bool is_v = works && !is_q && !is_k;
  const int v_unit = unit - q_units - k_units, v_head = v_unit / v_pieces, v_first = (v_unit - v_head * v_pieces) * 64 * PJ;
  const int len = is_v ? min(64 * PJ, p.vdim - v_first) : p.dim;
  const int ch0 = is_v ? (q_units + k_units) * p.dim + v_head * p.vdim + v_first : unit * p.dim;
  const float* weight = is_q ? p.q_weight : (is_k ? p.k_weight : nullptr);
  pdl_trigger();
  float2 w[TAPS > 0 ? TAPS : 1][PJ];
  float2 gain[PJ];
  if (works) {
#pragma unroll
    for (int j = 0; j < PJ; ++j) {
      const int c = 2 * (lane + 32 * j);
      gain[j] = make_float2(1.f, 1.f);
      if (weight != nullptr && c < len) gain[j] = make_float2(weight[c], c + 1 < len ? weight[c + 1] : 0.f);
      if (TAPS > 0) {
#pragma unroll
        for (int k = 0; k < TAPS; ++k)
          w[k][j] = c < len ? make_float2(p.conv[(long long)k * channels + ch0 + c],
                                          c + 1 < len ? p.conv[(long long)k * channels + ch0 + c + 1] : 0.f)
                            : make_float2(0.f, 0.f);
      }
    }
  }
  pdl_wait();
  const int t_first = blockIdx.x * RUN, t_end = min(p.n_tokens, t_first + RUN), half = p.rot_dims >> 1;
  for (int i = threadIdx.x; i < (t_end - t_first) * half; i += DA_PREP_WARPS * 32) {
    const int t = i / half, pair = i - t * half;
    float sn, cs;
    sincosf((float)p.positions[t_first + t] * p.inv_freq[pair], &sn, &cs);
    turn[i] = make_float2(cs * p.rot_size, sn * p.rot_size);
  }
  // where the run's tokens lie: lane i looks up token i, so that the look-ups of a run wait for one another once
  int at_r = 0, at_slot = 0, at_row = 0;
  if (lane < t_end - t_first) {
    const int t = t_first + lane, seq = p.token_seq[t], pos = p.positions[t];
    at_r = t - p.seq_start[seq];
    at_slot = p.slots[seq];
    const int lp = pos / p.page_size;
    at_row = p.table[(long long)seq * p.table_stride + (lp % p.table_len)] * p.n_kv_heads * p.page_size + pos - lp * p.page_size;
  }
  __syncthreads();
  if (!works) return;
  const T* src = reinterpret_cast<const T*>(p.proj) + ch0;
  const bool word = p.pairs_ok != 0;
  const int dkv = 2 * p.dim + p.vdim;
  float2 past[TAPS > 1 ? TAPS - 1 : 1][PJ];        // the inputs before the token, the newest last
  float2 own[RUN][PJ];                             // the run's inputs
#pragma unroll
  for (int i = 0; i < RUN; ++i)
#pragma unroll
    for (int j = 0; j < PJ; ++j) {
      const int c = 2 * (lane + 32 * j);
      own[i][j] = t_first + i < t_end && c < len ? da_pair<T>(src + (long long)(t_first + i) * p.row_stride + c, c + 1 < len, word)
                                                 : make_float2(0.f, 0.f);
    }
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    const int t = t_first + i;
    if (t >= t_end) break;
    const int r = __shfl_sync(0xffffffffu, at_r, i), slot = __shfl_sync(0xffffffffu, at_slot, i);
    const long long pool_row = __shfl_sync(0xffffffffu, at_row, i);
    float* kept = p.state + (long long)slot * (taps - 1) * channels + ch0;
    float2 y[PJ];
    float ss = 0.f;
    // the input `back` tokens before the sequence's r-th of this step, at channel c
    auto input = [&](int back, int c) {
      const bool two = c + 1 < len;
      if (back <= r) return da_pair<T>(src + (long long)(t - back) * p.row_stride + c, two, word);
      const float* cell = kept + (long long)(taps - 1 + r - back) * channels + c;
      return make_float2(cell[0], two ? cell[1] : 0.f);
    };
#pragma unroll
    for (int j = 0; j < PJ; ++j) {
      const int c = 2 * (lane + 32 * j);
      const bool one = c < len;
      float2 acc = make_float2(0.f, 0.f);
      const float2 u = own[i][j];
      if (TAPS > 0) {
        if (TAPS > 1 && (i == 0 || r == 0)) {
#pragma unroll
          for (int k = 0; k < TAPS - 1; ++k) past[k][j] = one ? input(TAPS - 1 - k, c) : make_float2(0.f, 0.f);
        }
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k) {
          acc.x = fmaf(w[k][j].x, past[k][j].x, acc.x);
          acc.y = fmaf(w[k][j].y, past[k][j].y, acc.y);
        }
        acc.x = fmaf(w[TAPS > 0 ? TAPS - 1 : 0][j].x, u.x, acc.x);
        acc.y = fmaf(w[TAPS > 0 ? TAPS - 1 : 0][j].y, u.y, acc.y);
#pragma unroll
        for (int k = 0; k + 1 < TAPS - 1; ++k) past[k][j] = past[k + 1][j];
        if (TAPS > 1) past[TAPS > 1 ? TAPS - 2 : 0][j] = u;
      } else if (one) {
        for (int k = 0; k < taps; ++k) {
          const float* wk = p.conv + (long long)k * channels + ch0 + c;
          const float2 x = k == taps - 1 ? u : input(taps - 1 - k, c);
          acc.x = fmaf(wk[0], x.x, acc.x);
          acc.y = fmaf(c + 1 < len ? wk[1] : 0.f, x.y, acc.y);
        }
      }
      y[j] = acc;
      ss = fmaf(acc.x, acc.x, fmaf(acc.y, acc.y, ss));
      if (p.shift_state && one && taps > 1) {
        // one token a sequence: nobody else reads these channels of the sequence's state
        for (int k = 0; k + 1 < taps - 1; ++k) {
          kept[(long long)k * channels + c] = kept[(long long)(k + 1) * channels + c];
          if (c + 1 < len) kept[(long long)k * channels + c + 1] = kept[(long long)(k + 1) * channels + c + 1];
        }
        kept[(long long)(taps - 2) * channels + c] = u.x;
        if (c + 1 < len) kept[(long long)(taps - 2) * channels + c + 1] = u.y;
      }
    }
    T* dst;
    if (is_q) {
      dst = reinterpret_cast<T*>(p.q_out) + (long long)t * q_units * p.q_pad + (long long)unit * p.q_pad;
    } else {
      const int g = is_k ? (unit - q_units) >> 1 : v_head;
      dst = reinterpret_cast<T*>(p.pool) + (pool_row + (long long)g * p.page_size) * dkv +
            (is_k ? ((unit - q_units) & 1) * p.dim : 2 * p.dim + v_first);
    }
    const float inv = weight != nullptr ? 1.f / sqrtf(warp_sum(ss) / (float)len + p.eps) : 1.f;
#pragma unroll
    for (int j = 0; j < PJ; ++j) {
      const int c = 2 * (lane + 32 * j);
      if (c >= len) continue;
      float u = y[j].x * inv * gain[j].x, v = y[j].y * inv * gain[j].y;
      if (!is_v && c < p.rot_dims) {
        const float2 cs = turn[i * half + (c >> 1)];
        const float a = u * cs.x - v * cs.y;
        v = v * cs.x + u * cs.y;
        u = a;
      }
      da_store_pair(dst + c, u, v, c + 1 < len, word);
    }
    if (is_q)
      for (int c = len + lane; c < p.q_pad; c += 32) dst[c] = from_float<T>(0.f);
  }
}

// state[slot] <- the last taps - 1 inputs of the sequence after this step (steps in which some sequence brings several)
template <typename T>
__global__ void __launch_bounds__(256)
differential_state_kernel(const T* __restrict__ proj, long long row_stride, float* __restrict__ state,
                          const int* __restrict__ slots, const int* __restrict__ seq_start, int n_seqs, int channels, int taps) {
  pdl_trigger();
  pdl_wait();
  const int keep = taps - 1;
  const long long total = (long long)n_seqs * channels;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int seq = (int)(i / channels), c = (int)(i - (long long)seq * channels);
    const int first = seq_start[seq], n_new = seq_start[seq + 1] - first;
    float* cell = state + (long long)slots[seq] * keep * channels + c;
    for (int k = 0; k < keep; ++k) {          // (from the oldest on: what is read lies behind what has been written)
      const int r = n_new - keep + k;
      cell[(long long)k * channels] = r >= 0 ? to_float(proj[(long long)(first + r) * row_stride + c])
                                             : cell[(long long)(keep + r) * channels];
    }
  }
}

// 16 bytes of shared memory as numbers.
__device__ __forceinline__ void da_piece(const float* p, float (&o)[4]) {
  const float4 f = *reinterpret_cast<const float4*>(p);
  o[0] = f.x; o[1] = f.y; o[2] = f.z; o[3] = f.w;
}
__device__ __forceinline__ void da_piece(const __nv_bfloat16* p, float (&o)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(h[i]);
    o[2 * i] = f.x;
    o[2 * i + 1] = f.y;
  }
}
__device__ __forceinline__ void da_copy16(void* smem, const void* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem) : "memory");
}

struct TwoMapArgs {
  const void* q;                    // rows of 2 heads dim_pad channels
  long long q_row_stride;
  int q_pad;
  const void* pool;
  const int *table, *token_seq, *positions;
  int table_stride, table_len, page_size;
  float* out;                       // n_splits == 1: [tokens][2 heads][vdim]; else parts [tokens][2 heads][splits][vdim + 2]
  int n_heads, n_kv_heads, head_tiles, n_splits, dim, vdim, ks;
  float scale;
};

// grid (key heads x head tiles x splits, tokens).  A block holds one token's rows of ROWS / 2 query heads of one key head
// (row 2 i + m: map m of the tile's i-th head); its warps share the split's key tiles, warp w taking tiles w, w + W, ...,
// each into shared memory of its own, so no block barrier stands between tiles.  For the scores a lane is a key and holds
// all rows' scores, for the value sum a lane is a set of value channels; each warp keeps a running maximum and sum a row,
// and the warps meet at the end in warp order.
template <typename T, int ROWS, int DVL>
__global__ void __launch_bounds__(256) two_map_attention_kernel(TwoMapArgs p) {
  extern __shared__ __align__(16) float smem[];
  const int n_warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int dim = p.dim, vdim = p.vdim, ks = p.ks, dkv = 2 * dim + vdim;
  float* q_s = smem;                                                                // [dim][ROWS]
  const int tile_words = (DA_TK * (ks + vdim) * (int)sizeof(T) + 15) / 16 * 4;
  T* k_s = reinterpret_cast<T*>(q_s + (ROWS * dim + 3) / 4 * 4 + (size_t)warp * tile_words);   // this warp's [DA_TK][ks]: both keys
  T* v_s = k_s + DA_TK * ks;                                                        // this warp's [DA_TK][vdim]
  pdl_trigger();
  pdl_wait();
  const long long token = blockIdx.y;
  const int split = blockIdx.x % p.n_splits, rest = blockIdx.x / p.n_splits;
  const int g = rest / p.head_tiles, head_tile = rest - g * p.head_tiles;
  const int group_heads = p.n_heads / p.n_kv_heads;
  const int h0 = g * group_heads + head_tile * (ROWS / 2);
  const int rows = 2 * min(ROWS / 2, (g + 1) * group_heads - h0);
  const int seq = p.token_seq[token], pos = p.positions[token];
  float acc[ROWS][DVL], top[ROWS], sum[ROWS];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    top[r] = -INFINITY;
    sum[r] = 0.f;
#pragma unroll
    for (int j = 0; j < DVL; ++j) acc[r][j] = 0.f;
  }
  const int n_tiles = pos / DA_TK + 1, per_split = (n_tiles + p.n_splits - 1) / p.n_splits;
  const int tile_end = min(n_tiles, (split + 1) * per_split);
  constexpr int V = 16 / (int)sizeof(T);
  const bool pieces_ok = dim % V == 0 && vdim % V == 0 && (reinterpret_cast<unsigned long long>(p.pool) & 15) == 0;
  // (a tile never straddles a page, and a key head's rows lie one after another in it.  Positions past the token's own hold
  // finite numbers of whoever had the page before: their weights are zero)
  auto fetch = [&](int tile) {
    const int j0 = tile * DA_TK, lp = j0 / p.page_size;
    const long long page = p.table[(long long)seq * p.table_stride + (lp % p.table_len)];
    const T* src = reinterpret_cast<const T*>(p.pool) + ((page * p.n_kv_heads + g) * p.page_size + (j0 - lp * p.page_size)) * dkv;
    if (pieces_ok) {
      const int per_row = dkv / V, n_pieces = DA_TK * per_row;
      for (int i = lane; i < n_pieces; i += 32) {
        const int kk = i / per_row, d0 = (i - kk * per_row) * V;
        da_copy16(d0 < 2 * dim ? k_s + kk * ks + d0 : v_s + kk * vdim + (d0 - 2 * dim), src + (long long)i * V);
      }
    } else {
      for (int i = lane; i < DA_TK * dkv; i += 32) {
        const int kk = i / dkv, d = i - kk * dkv;
        if (d < 2 * dim) k_s[kk * ks + d] = src[i]; else v_s[kk * vdim + d - 2 * dim] = src[i];
      }
    }
  };
  const int tile_first = split * per_split + warp;
  if (tile_first < tile_end) fetch(tile_first);          // (the queries are laid out while the first tile is on its way)
  const T* q = reinterpret_cast<const T*>(p.q) + token * p.q_row_stride + (long long)2 * h0 * p.q_pad;
  for (int i = threadIdx.x; i < ROWS * dim; i += blockDim.x) {
    const int r = i / dim, d = i - r * dim;
    q_s[d * ROWS + r] = r < rows ? to_float(q[(long long)r * p.q_pad + d]) : 0.f;
  }
  __syncthreads();
  for (int tile = tile_first; tile < tile_end; tile += n_warps) {
    const int j0 = tile * DA_TK;
    if (tile != tile_first) {
      __syncwarp();          // the lanes are done with the tile before
      fetch(tile);
    }
    asm volatile("cp.async.wait_all;\n" ::: "memory");
    __syncwarp();
    float s[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) s[r] = 0.f;
    const T* krow = k_s + lane * ks;
    auto take = [&](int d, float k1, float k2) {
      const float* qd = q_s + d * ROWS;
      if (ROWS % 4 == 0) {
#pragma unroll
        for (int r4 = 0; r4 < ROWS / 4; ++r4) {
          const float4 qv = *reinterpret_cast<const float4*>(qd + 4 * r4);
          s[4 * r4 + 0] = fmaf(qv.x, k1, s[4 * r4 + 0]);
          s[4 * r4 + 1] = fmaf(qv.y, k2, s[4 * r4 + 1]);
          s[4 * r4 + 2] = fmaf(qv.z, k1, s[4 * r4 + 2]);
          s[4 * r4 + 3] = fmaf(qv.w, k2, s[4 * r4 + 3]);
        }
      } else {
#pragma unroll
        for (int r = 0; r < ROWS; r += 2) {
          s[r] = fmaf(qd[r], k1, s[r]);
          s[r + 1] = fmaf(qd[r + 1], k2, s[r + 1]);
        }
      }
    };
    int d = 0;
    if (pieces_ok) {
#pragma unroll 2
      for (; d < dim; d += V) {
        float k1[V], k2[V];
        da_piece(krow + d, k1);
        da_piece(krow + dim + d, k2);
#pragma unroll
        for (int u = 0; u < V; ++u) take(d + u, k1[u], k2[u]);
      }
    }
    for (; d < dim; ++d) take(d, to_float(krow[d]), to_float(krow[dim + d]));
    const bool seen = j0 + lane <= pos;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      const float x = seen ? s[r] * p.scale : -INFINITY;
      const float m_new = fmaxf(top[r], warp_max(x));          // (key j0 is always seen: finite)
      const float aged = expf(top[r] - m_new);                 // 0 for the first tile
      s[r] = seen ? expf(x - m_new) : 0.f;
      sum[r] = sum[r] * aged + s[r];                           // this lane's keys; the lanes meet at the end
      top[r] = m_new;
#pragma unroll
      for (int j = 0; j < DVL; ++j) acc[r][j] *= aged;
    }
    const int kk_end = min(DA_TK, pos - j0 + 1);
    for (int kk = 0; kk < kk_end; ++kk) {
      float pk[ROWS];
#pragma unroll
      for (int r = 0; r < ROWS; ++r) pk[r] = __shfl_sync(0xffffffffu, s[r], kk);
#pragma unroll
      for (int j = 0; j < DVL; ++j) {
        const int c = lane + 32 * j;
        const float v = c < vdim ? to_float(v_s[kk * vdim + c]) : 0.f;
#pragma unroll
        for (int r = 0; r < ROWS; ++r) acc[r][j] = fmaf(pk[r], v, acc[r][j]);
      }
    }
  }
  // the warps' results, joined in warp order (the tiles' shared memory is free now)
  __syncthreads();
  float* sums = q_s + (ROWS * dim + 3) / 4 * 4;                // [n_warps][ROWS][vdim + 2]
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    float* cell = sums + ((size_t)warp * ROWS + r) * (vdim + 2);
#pragma unroll
    for (int j = 0; j < DVL; ++j) {
      const int c = lane + 32 * j;
      if (c < vdim) cell[c] = acc[r][j];
    }
    const float l = warp_sum(sum[r]);
    if (lane == 0) {
      cell[vdim] = top[r];
      cell[vdim + 1] = l;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < rows * (vdim + 2); i += blockDim.x) {
    const int r = i / (vdim + 2), c = i - r * (vdim + 2);
    const float* cell = sums + (size_t)r * (vdim + 2);
    const size_t step = (size_t)ROWS * (vdim + 2);
    float high = -INFINITY;
    for (int w = 0; w < n_warps; ++w) high = fmaxf(high, cell[w * step + vdim]);
    float total = 0.f, denom = 0.f;
    for (int w = 0; w < n_warps; ++w) {
      const float m = cell[w * step + vdim];
      const float f = m == -INFINITY ? 0.f : expf(m - high);
      denom = fmaf(f, cell[w * step + vdim + 1], denom);
      if (c < vdim) total = fmaf(f, cell[w * step + c], total);
    }
    const long long row = token * 2 * p.n_heads + 2 * h0 + r;
    if (p.n_splits == 1) {
      if (c < vdim) p.out[row * vdim + c] = total / denom;
    } else {
      p.out[(row * p.n_splits + split) * (vdim + 2) + c] = c < vdim ? total : (c == vdim ? high : denom);
    }
  }
}

// A warp a (token, head).  parts: as two_map_attention leaves them for n_splits.
template <typename T, int DVL>
__global__ void __launch_bounds__(128)
differential_combine_kernel(const float* __restrict__ parts, int n_splits, const float* __restrict__ share, float gain,
                            float eps, T* __restrict__ out, long long out_row_stride, long long items, int n_heads, int vdim) {
  pdl_trigger();
  pdl_wait();
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= items) return;
  const int lane = threadIdx.x & 31;
  const long long token = item / n_heads;
  const int head = (int)(item - token * n_heads);
  float o[2][DVL];
  const long long row = token * 2 * n_heads + 2 * head;          // the second map's row follows
  if (n_splits == 1) {
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int j = 0; j < DVL; ++j) {
        const int c = lane + 32 * j;
        o[m][j] = c < vdim ? parts[(row + m) * vdim + c] : 0.f;
      }
  } else {
    const int step = vdim + 2;
    const float* src = parts + row * n_splits * step;
    const long long second = (long long)n_splits * step;
    float w[2][DA_MAX_SPLITS / 32], l[2][DA_MAX_SPLITS / 32], denom[2] = {0.f, 0.f};
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int i = 0; i < DA_MAX_SPLITS / 32; ++i) {
        const int s = lane + 32 * i;
        w[m][i] = s < n_splits ? src[m * second + (long long)s * step + vdim] : -INFINITY;
        l[m][i] = s < n_splits ? src[m * second + (long long)s * step + vdim + 1] : 0.f;
      }
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      float high = -INFINITY;
#pragma unroll
      for (int i = 0; i < DA_MAX_SPLITS / 32; ++i) high = fmaxf(high, w[m][i]);
      high = warp_max(high);
#pragma unroll
      for (int i = 0; i < DA_MAX_SPLITS / 32; ++i) {
        w[m][i] = w[m][i] == -INFINITY ? 0.f : expf(w[m][i] - high);
        denom[m] = fmaf(w[m][i], l[m][i], denom[m]);
      }
      denom[m] = warp_sum(denom[m]);
#pragma unroll
      for (int j = 0; j < DVL; ++j) o[m][j] = 0.f;
    }
#pragma unroll 4
    for (int s = 0; s < n_splits; ++s) {
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const float f = __shfl_sync(0xffffffffu, s < 32 ? w[m][0] : w[m][DA_MAX_SPLITS / 32 - 1], s & 31);
#pragma unroll
        for (int j = 0; j < DVL; ++j) {
          const int c = lane + 32 * j;
          if (c < vdim) o[m][j] = fmaf(f, src[m * second + (long long)s * step + c], o[m][j]);
        }
      }
    }
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int j = 0; j < DVL; ++j) o[m][j] /= denom[m];
  }
  const float lambda = share[0];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < DVL; ++j) {
    o[0][j] -= lambda * o[1][j];
    ss = fmaf(o[0][j], o[0][j], ss);
  }
  const float f = gain / sqrtf(warp_sum(ss) / (float)vdim + eps);
#pragma unroll
  for (int j = 0; j < DVL; ++j) {
    const int c = lane + 32 * j;
    if (c < vdim) out[token * out_row_stride + (long long)head * vdim + c] = from_float<T>(o[0][j] * f);
  }
}

// (a warp takes one token in steps of few tokens, else as many as its registers hold the inputs of)
template <typename T, int TAPS>
static int launch_differential_prep(const DiffPrepArgs& p, cudaStream_t stream) {
#define BT_DP_RUN(PJ, RUN)                                                                                              \
  do {                                                                                                                  \
    const int units = 2 * (p.n_heads + p.n_kv_heads) + p.n_kv_heads * ((p.vdim + 64 * PJ - 1) / (64 * PJ));             \
    const dim3 grid((p.n_tokens + RUN - 1) / RUN, (units + DA_PREP_WARPS - 1) / DA_PREP_WARPS);                         \
    auto kernel = differential_prep_kernel<T, TAPS, PJ, RUN>;                                                           \
    BT_PDL_OK("differential_prep", launch_pdl(kernel, grid, dim3(DA_PREP_WARPS * 32),                                   \
                                              (size_t)RUN * (p.rot_dims / 2) * sizeof(float2), stream, 1, p));          \
  } while (0)
#define BT_DP(PJ, RUN)                                                                                                  \
  do {                                                                                                                  \
    if (p.n_tokens <= 256) BT_DP_RUN(PJ, 1); else BT_DP_RUN(PJ, RUN);                                                   \
  } while (0)
  if (p.dim <= 64) BT_DP(1, 8);
  else if (p.dim <= 128) BT_DP(2, 4);
  else BT_DP(4, 2);
#undef BT_DP
#undef BT_DP_RUN
  return 0;
}

template <typename T>
static int run_differential_prep(const DiffPrepArgs& p, int n_seqs, cudaStream_t stream) {
  int rc;
  switch (p.taps) {
    case 3: rc = launch_differential_prep<T, 3>(p, stream); break;
    case 4: rc = launch_differential_prep<T, 4>(p, stream); break;
    default: rc = launch_differential_prep<T, 0>(p, stream);
  }
  if (rc != 0 || p.taps == 1 || p.shift_state) return rc;
  const int channels = 2 * (p.n_heads + p.n_kv_heads) * p.dim + p.n_kv_heads * p.vdim;
  const long long blocks = ((long long)n_seqs * channels + 255) / 256;
  BT_PDL_OK("differential_state", launch_pdl(differential_state_kernel<T>, dim3((unsigned)(blocks < 2368 ? blocks : 2368)),
                                             dim3(256), 0, stream, 1, (const T*)p.proj, p.row_stride, p.state, p.slots,
                                             p.seq_start, n_seqs, channels, p.taps));
  return 0;
}

// Rows (a map of a query head) a block holds, and its warps and shared memory.
struct TwoMapShape { int rows, head_tiles, warps, ks; size_t smem; };
static TwoMapShape two_map_shape(int group_heads, int dim, int vdim, int elem) {
  TwoMapShape s;
  s.rows = group_heads <= 1 ? 2 : (group_heads <= 2 ? 4 : 8);
  s.head_tiles = (group_heads + s.rows / 2 - 1) / (s.rows / 2);
  // a key row's length in shared memory: whole 16-byte pieces, an odd number of them, so that the eight lanes of a 16-byte
  // read meet every bank once
  const int piece = 16 / elem;
  s.ks = (2 * dim + piece - 1) / piece * piece;
  if ((s.ks / piece) % 2 == 0) s.ks += piece;
  const size_t tile_words = ((size_t)DA_TK * (s.ks + vdim) * elem + 15) / 16 * 4;
  auto bytes = [&](int w) {
    const size_t tiles = (size_t)w * tile_words, sums = (size_t)w * s.rows * (vdim + 2);
    return (((size_t)s.rows * dim + 3) / 4 * 4 + (tiles > sums ? tiles : sums)) * sizeof(float);
  };
  s.warps = 4;
  while (s.warps > 1 && bytes(s.warps) > 160 * 1024) s.warps >>= 1;
  s.smem = bytes(s.warps);
  return s;
}

template <typename T>
static int launch_two_map(TwoMapArgs p, int n_tokens, cudaStream_t stream) {
  const TwoMapShape s = two_map_shape(p.n_heads / p.n_kv_heads, p.dim, p.vdim, (int)sizeof(T));
  BT_CHECK(s.smem <= 200 * 1024, "two_map_attention: heads of 2 x %d + %d channels need %zu bytes of shared memory", p.dim,
           p.vdim, s.smem);
  p.head_tiles = s.head_tiles;
  p.ks = s.ks;
  const dim3 grid(p.n_kv_heads * s.head_tiles * p.n_splits, n_tokens), block(s.warps * 32);
#define BT_TM_ROWS(ROWS, DVL)                                                                                         \
  do {                                                                                                                \
    auto kernel = two_map_attention_kernel<T, ROWS, DVL>;                                                             \
    if (s.smem > 48 * 1024) {                                                                                         \
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s.smem);         \
      BT_CHECK(e == cudaSuccess, "two_map_attention: cannot reserve %zu bytes of shared memory", s.smem);             \
    }                                                                                                                 \
    BT_PDL_OK("two_map_attention", launch_pdl(kernel, grid, block, s.smem, stream, 1, p));                            \
  } while (0)
#define BT_TM(DVL)                                                                                                    \
  do {                                                                                                                \
    if (s.rows == 2) BT_TM_ROWS(2, DVL); else if (s.rows == 4) BT_TM_ROWS(4, DVL); else BT_TM_ROWS(8, DVL);           \
  } while (0)
  if (p.vdim <= 32) BT_TM(1);
  else if (p.vdim <= 64) BT_TM(2);
  else if (p.vdim <= 128) BT_TM(4);
  else BT_TM(8);
#undef BT_TM
#undef BT_TM_ROWS
  return 0;
}

template <typename T>
static int launch_differential_combine(const float* parts, int n_splits, const float* share, float gain, float eps, T* out,
                                       long long out_row_stride, int n_tokens, int n_heads, int vdim, cudaStream_t stream) {
  const long long items = (long long)n_tokens * n_heads;
  const dim3 grid((unsigned)((items + 3) / 4)), block(128);
#define BT_DC(DVL)                                                                                                    \
  BT_PDL_OK("differential_combine", launch_pdl(differential_combine_kernel<T, DVL>, grid, block, 0, stream, 1, parts, n_splits, \
                                               share, gain, eps, out, out_row_stride, items, n_heads, vdim))
  if (vdim <= 64) BT_DC(2);
  else if (vdim <= 128) BT_DC(4);
  else BT_DC(8);
#undef BT_DC
  return 0;
}

}  // namespace bt

// proj: rows of the step's tokens as DiffPrepArgs says; conv [taps][channels] 32-bit; q_weight, k_weight [dim] 32-bit (both
// null: queries and keys are not normed).  max_new: no sequence brings more tokens than this.
extern "C" int bt_differential_prep(const void* proj, long long row_stride, const float* conv, float* state, const int* slots,
                                    const int* seq_start, const int* token_seq, const int* positions, const float* q_weight,
                                    const float* k_weight, float eps, const float* inv_freq, int rot_dims, float rot_size,
                                    int taps, const int* table, int table_stride, int table_len, int page_size, void* pool,
                                    long long pool_pages, void* q_out, int q_pad, int n_tokens, int n_seqs, int max_new, int n_heads, int n_kv_heads,
                                    int dim, int vdim, int dtype, cudaStream_t stream) {
  using namespace bt;
  // (a pool's rows are counted in 32 bits)
  BT_CHECK(n_tokens >= 0 && n_heads > 0 && n_kv_heads > 0 && n_heads % n_kv_heads == 0 && dim > 0 && dim <= 256 && vdim > 0 &&
               vdim <= 256 && pool_pages > 0 && pool_pages * n_kv_heads * page_size < (1ll << 31) && rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim && taps >= 1 && taps <= DA_MAX_TAPS &&
               q_pad >= dim,
           "differential_prep: bad sizes heads=%d kv_heads=%d dim=%d vdim=%d (up to 256) rot_dims=%d taps=%d (up to %d)", n_heads,
           n_kv_heads, dim, vdim, rot_dims, taps, DA_MAX_TAPS);
  if (n_tokens == 0) return 0;
  const int elem = dtype == kF32 ? 4 : 2;
  auto pairs = [&](const void* ptr) { return (unsigned long long)ptr % (2 * elem) == 0; };
  const int words = row_stride % 2 == 0 && dim % 2 == 0 && vdim % 2 == 0 && q_pad % 2 == 0 && pairs(proj) && pairs(pool) && pairs(q_out);
  DiffPrepArgs p{proj, row_stride, conv, state, slots, seq_start, token_seq, positions, table, q_weight, k_weight, inv_freq, eps,
                 rot_size, rot_dims, taps, table_stride, table_len, page_size, pool, q_out, n_tokens, n_heads, n_kv_heads, dim,
                 vdim, q_pad, max_new == 1, words};
  if (dtype == kF32) return run_differential_prep<float>(p, n_seqs, stream);
  if (dtype == kBF16) return run_differential_prep<__nv_bfloat16>(p, n_seqs, stream);
  return fail("differential_prep: unknown dtype %d", dtype);
}

// Both maps of every token over the pages up to its own position.  q: rows of 2 heads q_pad channels.
extern "C" int bt_two_map_attention(const void* q, long long q_row_stride, int q_pad, const void* pool, const int* table,
                                    int table_stride, int table_len, int page_size, const int* token_seq,
                                    const int* positions, float* out, int n_tokens, int n_heads, int n_kv_heads, int dim,
                                    int vdim, float scale, int n_splits, int dtype, cudaStream_t stream) {
  using namespace bt;
  BT_CHECK(n_tokens >= 0 && n_heads > 0 && n_kv_heads > 0 && n_heads % n_kv_heads == 0 && dim > 0 && dim <= 256 && vdim > 0 &&
               vdim <= 256 && n_splits >= 1 && n_splits <= DA_MAX_SPLITS && page_size % DA_TK == 0,
           "two_map_attention: bad sizes heads=%d kv_heads=%d dim=%d vdim=%d (up to 256) splits=%d", n_heads, n_kv_heads, dim,
           vdim, n_splits);
  TwoMapArgs p{q, q_row_stride, q_pad, pool, table, token_seq, positions, table_stride, table_len, page_size, out, n_heads,
               n_kv_heads, 0, n_splits, dim, vdim, 0, scale};
  const long long step = q_row_stride, out_step = 2ll * n_heads * (n_splits > 1 ? n_splits * (vdim + 2) : vdim);
  // (a launch's second grid axis ends at 65,535)
  for (int t0 = 0; t0 < n_tokens; t0 += 65535) {
    const int n = n_tokens - t0 < 65535 ? n_tokens - t0 : 65535;
    TwoMapArgs part = p;
    part.q = (const char*)q + (long long)t0 * step * (dtype == kF32 ? 4 : 2);
    part.token_seq = token_seq + t0;
    part.positions = positions + t0;
    part.out = out + t0 * out_step;
    int rc;
    if (dtype == kF32) rc = launch_two_map<float>(part, n, stream);
    else if (dtype == kBF16) rc = launch_two_map<__nv_bfloat16>(part, n, stream);
    else return fail("two_map_attention: unknown dtype %d", dtype);
    if (rc != 0) return rc;
  }
  return 0;
}

// out[t, h] = o / sqrt(mean(o^2) + eps) * gain, o = first map's result - share[0] * the second's.
extern "C" int bt_differential_combine(const float* parts, int n_splits, const float* share, float gain, float eps, void* out,
                                       long long out_row_stride, int n_tokens, int n_heads, int vdim, int dtype,
                                       cudaStream_t stream) {
  using namespace bt;
  BT_CHECK(n_tokens >= 0 && n_heads > 0 && vdim > 0 && vdim <= 256 && n_splits >= 1 && n_splits <= DA_MAX_SPLITS,
           "differential_combine: bad sizes heads=%d vdim=%d splits=%d", n_heads, vdim, n_splits);
  if (n_tokens == 0) return 0;
  if (dtype == kF32)
    return launch_differential_combine<float>(parts, n_splits, share, gain, eps, (float*)out, out_row_stride, n_tokens, n_heads,
                                              vdim, stream);
  if (dtype == kBF16)
    return launch_differential_combine<__nv_bfloat16>(parts, n_splits, share, gain, eps, (__nv_bfloat16*)out, out_row_stride,
                                                      n_tokens, n_heads, vdim, stream);
  return fail("differential_combine: unknown dtype %d", dtype);
}
