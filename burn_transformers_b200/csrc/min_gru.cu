// A gated average per channel, carried from token to token:
//
//   z_t = sigmoid(a_t + b_z),  v_t = u + 1/2 for u >= 0 and sigmoid(u) for u < 0 with u = x_t + b_x
//   S_t = (1 - z_t) S_(t-1) + z_t v_t
//   out_t = S_t * g_t sigmoid(g_t)
//
// a, x and g are `width` channels each of a token's projected row; nothing of them depends on S, so the map of a run of
// tokens, S -> A S + B, can be formed for all runs at once and the maps composed: (A1, B1) then (A2, B2) is (A1 A2,
// A2 B1 + B2).  All A lie in [0, 1] and all B are sums of positive numbers: nothing cancels and nothing overflows.
// Everything from the biases on is 32-bit; the result is rounded once.
//
//   few tokens    a thread per sequence and channel pair walks the step's tokens
//   long runs     one kernel: a cluster of up to 8 blocks owns a sequence's tokens for 32 * V channels; a warp holds
//                 MG_TOK tokens in registers (read once), a block MG_WARPS of them, the cluster all its blocks'.  The
//                 warps' maps are composed in shared memory, the blocks' maps are read by every block of the cluster
//                 through distributed shared memory; then each warp runs its tokens from the state that reaches it.
//                 A run longer than the cluster holds goes round in a loop that carries the state.
#include <cooperative_groups.h>

#include "common.cuh"

namespace bt {

namespace cg = cooperative_groups;

constexpr int MG_WARPS = 8, MG_TOK = 8, MG_MAX_CLUSTER = 8, MG_BLOCKS = 2;
constexpr int MG_FEW = 16;       // runs of at most this many tokens are walked by single threads

struct MinGruArgs {
  const void* proj;              // rows of `row_stride` elements: a at z_off, x at x_off, g at g_off
  long long row_stride;
  int z_off, x_off, g_off;
  const float* z_bias;           // [width] each
  const float* x_bias;
  float* state;                  // [slots, width]
  const int* slots;
  const int* seq_start;
  void* out;                     // rows of `out_stride` elements
  long long out_stride;
  int width;
};

// 32-bit rows take CUDA's full-precision functions; rows that come as bfloat16 (and leave rounded to it) the
// special-function unit's exponential and reciprocal, whose errors are a few units in the last place of 32-bit.
template <bool EXACT> __device__ __forceinline__ float exponential(float v) { return EXACT ? expf(v) : __expf(v); }
template <bool EXACT> __device__ __forceinline__ float quotient(float a, float b) { return EXACT ? a / b : __fdividef(a, b); }
// (exp(-v) may overflow to infinity: the quotient is then zero, which is the limit)
template <bool EXACT> __device__ __forceinline__ float logistic(float v) {
  return quotient<EXACT>(1.f, 1.f + exponential<EXACT>(-v));
}

// the map of one token: keep = 1 - z, add = z * v.  With e = exp(-|s|), z and 1 - z are 1 / (1 + e) and e / (1 + e), one
// or the other way round by the sign of s: neither is a difference of nearly equal numbers.
template <bool EXACT>
__device__ __forceinline__ void token_map(float s, float u, float& keep, float& add) {
  const float e = exponential<EXACT>(-fabsf(s)), big = quotient<EXACT>(1.f, 1.f + e), small = e * big;
  keep = s >= 0.f ? small : big;
  const float share = s >= 0.f ? big : small;
  add = share * (u >= 0.f ? u + 0.5f : logistic<EXACT>(u));
}

// V neighbouring channels as one access (V * sizeof(T) bytes; the host has checked the alignment), as they lie in memory
template <typename T, int V> struct Raw;
template <> struct Raw<float, 1> { float v; };
template <> struct Raw<float, 2> { float2 v; };
template <> struct Raw<__nv_bfloat16, 1> { __nv_bfloat16 v; };
template <> struct Raw<__nv_bfloat16, 2> { __nv_bfloat162 v; };

template <typename T, int V> __device__ __forceinline__ Raw<T, V> load_raw(const T* p) {
  return *reinterpret_cast<const Raw<T, V>*>(p);
}
__device__ __forceinline__ void unpack(const Raw<float, 1>& r, float (&o)[1]) { o[0] = r.v; }
__device__ __forceinline__ void unpack(const Raw<float, 2>& r, float (&o)[2]) { o[0] = r.v.x; o[1] = r.v.y; }
__device__ __forceinline__ void unpack(const Raw<__nv_bfloat16, 1>& r, float (&o)[1]) { o[0] = __bfloat162float(r.v); }
__device__ __forceinline__ void unpack(const Raw<__nv_bfloat16, 2>& r, float (&o)[2]) {
  const float2 f = __bfloat1622float2(r.v);
  o[0] = f.x; o[1] = f.y;
}
__device__ __forceinline__ void store_channels(float* p, const float (&o)[1]) { p[0] = o[0]; }
__device__ __forceinline__ void store_channels(float* p, const float (&o)[2]) {
  *reinterpret_cast<float2*>(p) = make_float2(o[0], o[1]);
}
__device__ __forceinline__ void store_channels(__nv_bfloat16* p, const float (&o)[1]) { p[0] = __float2bfloat16_rn(o[0]); }
__device__ __forceinline__ void store_channels(__nv_bfloat16* p, const float (&o)[2]) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(o[0], o[1]);
}

template <typename T, int V>
__global__ void __launch_bounds__(64) min_gru_few_kernel(MinGruArgs p) {
  const int c = (blockIdx.x * 64 + threadIdx.x) * V, seq = blockIdx.y;
  constexpr bool EXACT = sizeof(T) == 4;
  const bool in = c < p.width;
  float zb[V], xb[V];
  unpack(load_raw<float, V>(p.z_bias + (in ? c : 0)), zb);
  unpack(load_raw<float, V>(p.x_bias + (in ? c : 0)), xb);
  pdl_trigger();
  pdl_wait();
  if (!in) return;
  const int first = p.seq_start[seq], last = p.seq_start[seq + 1];
  float* kept = p.state + (long long)p.slots[seq] * p.width + c;
  float s[V];
  unpack(load_raw<float, V>(kept), s);
  const T* row = reinterpret_cast<const T*>(p.proj) + (long long)first * p.row_stride + c;
  T* out = reinterpret_cast<T*>(p.out) + (long long)first * p.out_stride + c;
  for (int t = first; t < last; ++t, row += p.row_stride, out += p.out_stride) {
    float a[V], x[V], g[V], y[V];
    const Raw<T, V> ra = load_raw<T, V>(row + p.z_off), rx = load_raw<T, V>(row + p.x_off), rg = load_raw<T, V>(row + p.g_off);
    unpack(ra, a);
    unpack(rx, x);
    unpack(rg, g);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      float keep, add;
      token_map<EXACT>(a[i] + zb[i], x[i] + xb[i], keep, add);
      s[i] = fmaf(keep, s[i], add);
      y[i] = s[i] * (g[i] * logistic<EXACT>(g[i]));
    }
    store_channels(out, y);
  }
  store_channels(kept, s);
}

// The map S -> keep S + add of a run of tokens, for a lane's V channels.
template <int V> struct __align__(8 * V) RunMap { float keep[V], add[V]; };

template <int V> __device__ __forceinline__ void then(RunMap<V>& m, const RunMap<V>& next) {
#pragma unroll
  for (int i = 0; i < V; ++i) {
    m.add[i] = fmaf(next.keep[i], m.add[i], next.add[i]);
    m.keep[i] *= next.keep[i];
  }
}

// grid (channel groups * cluster, sequences), cluster blocks along x; block: MG_WARPS warps.
template <typename T, int V>
__global__ void __launch_bounds__(MG_WARPS * 32, MG_BLOCKS)
min_gru_scan_kernel(MinGruArgs p, int cluster_size) {
  constexpr int CH = 32 * V;
  constexpr bool EXACT = sizeof(T) == 4;
  __shared__ RunMap<V> warp_map[MG_WARPS][32];      // the warps' maps, then the map of all tokens before each warp's
  __shared__ RunMap<V> block_map[2][32];            // the block's map, by turns (peers read it)
  __shared__ float enter[32][V];                    // the state before the block's first token
  cg::cluster_group cluster = cg::this_cluster();
  const int rank = (int)cluster.block_rank();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c0 = (blockIdx.x / cluster_size) * CH + lane * V, seq = blockIdx.y;
  const bool in = c0 < p.width;
  const int c = in ? c0 : 0;             // (a lane behind the last channel computes the first one's and stores nothing)
  float zb[V], xb[V];
  unpack(load_raw<float, V>(p.z_bias + c), zb);
  unpack(load_raw<float, V>(p.x_bias + c), xb);
  pdl_trigger();
  pdl_wait();
  const int first = p.seq_start[seq], count = p.seq_start[seq + 1] - first;
  float* kept = p.state + (long long)p.slots[seq] * p.width + c;
  float s[V] = {};                       // (warp 0: the state before this round of the loop)
  if (warp == 0) unpack(load_raw<float, V>(kept), s);
  const T* rows = reinterpret_cast<const T*>(p.proj) + (long long)first * p.row_stride + c;
  T* outs = reinterpret_cast<T*>(p.out) + (long long)first * p.out_stride + c;
  const int round_tokens = cluster_size * MG_WARPS * MG_TOK;
  // all reads of a warp's tokens in flight together: no branch, a place behind the run's last token reads that one
  Raw<T, V> ra[MG_TOK], rx[MG_TOK], rg[MG_TOK];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int k = 0; k < MG_TOK; ++k) {
      const T* row = rows + (long long)min(t0 + k, count - 1) * p.row_stride;
      ra[k] = load_raw<T, V>(row + p.z_off);
      rx[k] = load_raw<T, V>(row + p.x_off);
      rg[k] = load_raw<T, V>(row + p.g_off);
    }
  };
  const int mine = (rank * MG_WARPS + warp) * MG_TOK;
  if (count > 0) fetch(mine);
  int turn = 0;
  for (int base = 0; base < count; base += round_tokens, turn ^= 1) {
    const int t0 = base + mine;
    float keep[MG_TOK][V], add[MG_TOK][V];
    Raw<T, V> gate[MG_TOK];
#pragma unroll
    for (int k = 0; k < MG_TOK; ++k) {
      float a[V], x[V];
      unpack(ra[k], a);
      unpack(rx[k], x);
      gate[k] = rg[k];
#pragma unroll
      for (int i = 0; i < V; ++i) {
        token_map<EXACT>(a[i] + zb[i], x[i] + xb[i], keep[k][i], add[k][i]);
        if (t0 + k >= count) {                   // (... and leaves the state as it is)
          keep[k][i] = 1.f;
          add[k][i] = 0.f;
        }
      }
    }
    if (base + round_tokens < count) fetch(t0 + round_tokens);      // (the next round's, while this one's maps meet)
    RunMap<V> m;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      m.keep[i] = keep[0][i];
      m.add[i] = add[0][i];
#pragma unroll
      for (int k = 1; k < MG_TOK; ++k) {
        m.add[i] = fmaf(keep[k][i], m.add[i], add[k][i]);
        m.keep[i] *= keep[k][i];
      }
    }
    warp_map[warp][lane] = m;
    __syncthreads();
    if (warp == 0) {
      RunMap<V> all = {};
#pragma unroll
      for (int i = 0; i < V; ++i) all.keep[i] = 1.f;
#pragma unroll
      for (int w = 0; w < MG_WARPS; ++w) {
        const RunMap<V> own = warp_map[w][lane];
        warp_map[w][lane] = all;
        then(all, own);
      }
      block_map[turn][lane] = all;
    }
    cluster.sync();                    // every block's map is there (and, block by block, the warps' prefixes)
    if (warp == 0) {
      RunMap<V> peer[MG_MAX_CLUSTER];
#pragma unroll
      for (int b = 0; b < MG_MAX_CLUSTER; ++b) {
#pragma unroll
        for (int i = 0; i < V; ++i) { peer[b].keep[i] = 1.f; peer[b].add[i] = 0.f; }
        if (b < cluster_size) peer[b] = *cluster.map_shared_rank(&block_map[turn][lane], b);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) {
#pragma unroll
        for (int b = 0; b < MG_MAX_CLUSTER; ++b) {
          if (b == rank) enter[lane][i] = s[i];
          s[i] = fmaf(peer[b].keep[i], s[i], peer[b].add[i]);
        }
      }
    }
    __syncthreads();
    const RunMap<V> before = warp_map[warp][lane];
    float st[V];
#pragma unroll
    for (int i = 0; i < V; ++i) st[i] = fmaf(before.keep[i], enter[lane][i], before.add[i]);
#pragma unroll
    for (int k = 0; k < MG_TOK; ++k) {
      float g[V], y[V];
      unpack(gate[k], g);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        st[i] = fmaf(keep[k][i], st[i], add[k][i]);
        y[i] = st[i] * (g[i] * logistic<EXACT>(g[i]));
      }
      if (in && t0 + k < count) store_channels(outs + (long long)(t0 + k) * p.out_stride, y);
    }
    __syncthreads();                   // (the next round writes the warps' maps and `enter` again)
  }
  if (rank == 0 && warp == 0 && in) store_channels(kept, s);
  cluster.sync();                      // nobody leaves while a peer may still read its map
}

template <typename T, int V>
static int launch_min_gru(const MinGruArgs& p, int n_seqs, int max_new, cudaStream_t stream) {
  if (max_new <= MG_FEW) {
    const dim3 grid((p.width + 64 * V - 1) / (64 * V), n_seqs);
    BT_PDL_OK("min_gru", launch_pdl(min_gru_few_kernel<T, V>, grid, dim3(64), 0, stream, 1, p));
    return 0;
  }
  int cluster = 1;
  while (cluster < MG_MAX_CLUSTER && cluster * MG_WARPS * MG_TOK < max_new) cluster *= 2;
  const dim3 grid((unsigned)((p.width + 32 * V - 1) / (32 * V) * cluster), n_seqs);
  BT_PDL_OK("min_gru", launch_pdl(min_gru_scan_kernel<T, V>, grid, dim3(MG_WARPS * 32), 0, stream, cluster, p, cluster));
  return 0;
}

}  // namespace bt

extern "C" int bt_min_gru(const void* proj, long long row_stride, int z_off, int x_off, int g_off, const float* z_bias,
                          const float* x_bias, float* state, const int* slots, const int* seq_start, void* out,
                          long long out_row_stride, int n_seqs, int width, int max_new, int dtype, cudaStream_t stream) {
  using namespace bt;
  BT_CHECK(width > 0 && width < (1 << 28) && n_seqs >= 0 && n_seqs <= 65535 && max_new >= 0 && z_off >= 0 && x_off >= 0 && g_off >= 0,
           "min_gru: bad sizes width=%d sequences=%d", width, n_seqs);
  BT_CHECK(dtype == kF32 || dtype == kBF16, "min_gru: unknown dtype %d", dtype);
  if (n_seqs == 0 || max_new == 0) return 0;
  MinGruArgs p;
  p.proj = proj; p.row_stride = row_stride; p.z_off = z_off; p.x_off = x_off; p.g_off = g_off;
  p.z_bias = z_bias; p.x_bias = x_bias; p.state = state; p.slots = slots; p.seq_start = seq_start;
  p.out = out; p.out_stride = out_row_stride; p.width = width;
  const unsigned pair = dtype == kF32 ? 8 : 4;
  auto at = [](const void* ptr, unsigned bytes) { return (unsigned long long)ptr % bytes == 0; };
  const bool pairs = width % 2 == 0 && row_stride % 2 == 0 && out_row_stride % 2 == 0 && z_off % 2 == 0 && x_off % 2 == 0 &&
                     g_off % 2 == 0 && at(proj, pair) && at(out, pair) && at(state, 8) && at(z_bias, 8) && at(x_bias, 8);
  if (dtype == kF32) return pairs ? launch_min_gru<float, 2>(p, n_seqs, max_new, stream) : launch_min_gru<float, 1>(p, n_seqs, max_new, stream);
  return pairs ? launch_min_gru<__nv_bfloat16, 2>(p, n_seqs, max_new, stream)
               : launch_min_gru<__nv_bfloat16, 1>(p, n_seqs, max_new, stream);
}
