// Gated linear attention: a recurrence over a 32-bit state per (sequence, head) whose decay is a number per KEY CHANNEL and
// token:
//
//     S_t = diag(a_t) S_(t-1) + k_t v_t^T        (S: dim x vdim, a_t: dim numbers in (0, 1])
//     o_t = S_t^T (q_t * q_scale)
//
// with a_t = exp(log_scale * dt_t), dt the caller's 32-bit rows [tokens][heads dim] (log_scale < 0 <= dt: a softplus of the
// negated gate's pre-activation, for instance).  q, k, v are channels of the step's projections, taken as they are.
// The state lives in `state[slot][head][dim][vdim]`; a sequence that starts finds zeros there.
//
// Token by token (gla_scan_kernel): a block owns value channels of one (sequence, head) and keeps its part of the state in
// registers for all tokens of the step; a value channel belongs to SPLIT adjacent lanes with DPT key channels each.
// A block that holds a whole head also divides the head's o by its root mean square, multiplies by a weight and by
// g * sigmoid(g), and writes the row that the output projection reads.
//
// Long runs go by chunks, further below.
#include "common.cuh"

namespace bt {

constexpr int GS_TOKENS = 16;  // tokens staged in shared memory at a time

// exp for decays: the special-function unit's form beside bfloat16 rows, the library's beside 32-bit rows
template <typename T> __device__ __forceinline__ float gla_exp(float x) { return __expf(x); }
template <> __device__ __forceinline__ float gla_exp<float>(float x) { return expf(x); }

struct GlaNorm {               // weight null: the block leaves o in `out`
  const float* weight;         // [vdim], shared by the heads
  float eps;
  int g_off;
  void* mixed;
  long long mixed_row_stride;
};

template <typename T, int DPT, int SPLIT>
__global__ void __launch_bounds__(512)
gla_scan_kernel(const T* __restrict__ proj, long long row_stride, int q_off, int k_off, int v_off, float q_scale,
                const float* __restrict__ dt, float log_scale, float* __restrict__ state, const int* __restrict__ slots,
                const int* __restrict__ seq_start, float* __restrict__ out, long long out_row_stride, int n_heads, int dim,
                int vdim, int cols, GlaNorm norm) {
  extern __shared__ float sm[];
  float* q_s = sm;                          // [GS_TOKENS][dim]
  float* k_s = q_s + GS_TOKENS * dim;       // [GS_TOKENS][dim]
  float* a_s = k_s + GS_TOKENS * dim;       // [GS_TOKENS][dim]
  float* v_s = a_s + GS_TOKENS * dim;       // [GS_TOKENS][cols]; with a norm, o takes its place
  pdl_trigger();
  pdl_wait();
  const int seq = blockIdx.z, head = blockIdx.y, col0 = blockIdx.x * cols;
  const int first = seq_start[seq], n_new = seq_start[seq + 1] - first;
  const int part = threadIdx.x % SPLIT, col_local = threadIdx.x / SPLIT;
  const int col = col0 + col_local;
  const bool owns = col_local < cols && col < vdim;
  const int d0 = part * DPT;
  float* s_base = state + (((long long)slots[seq] * n_heads + head) * dim) * vdim;
  float s[DPT];
#pragma unroll
  for (int i = 0; i < DPT; ++i) s[i] = owns && d0 + i < dim ? s_base[(long long)(d0 + i) * vdim + col] : 0.f;
  for (int t0 = 0; t0 < n_new; t0 += GS_TOKENS) {
    const int nt = min(GS_TOKENS, n_new - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * dim; i += blockDim.x) {
      const int t = i / dim, d = i - t * dim;
      const long long row = first + t0 + t;
      const T* src = proj + row * row_stride + (long long)head * dim + d;
      q_s[i] = to_float(src[q_off]) * q_scale;
      k_s[i] = to_float(src[k_off]);
      a_s[i] = gla_exp<T>(dt[(row * n_heads + head) * dim + d] * log_scale);
    }
    for (int i = threadIdx.x; i < nt * cols; i += blockDim.x) {
      const int t = i / cols, c = i - t * cols;
      v_s[i] = col0 + c < vdim
                   ? to_float(proj[(long long)(first + t0 + t) * row_stride + v_off + (long long)head * vdim + col0 + c]) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float v = col_local < cols ? v_s[t * cols + col_local] : 0.f;
      const float* kt = k_s + t * dim + d0;
      const float* qt = q_s + t * dim + d0;
      const float* at = a_s + t * dim + d0;
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < DPT; ++i) {
        if (d0 + i < dim) {
          s[i] = fmaf(at[i], s[i], kt[i] * v);
          o = fmaf(s[i], qt[i], o);
        }
      }
#pragma unroll
      for (int x = 1; x < SPLIT; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
      if (owns && part == 0) {
        // (a column's v of this token was read by its own lanes above, before the shuffles)
        if (norm.weight != nullptr) v_s[t * cols + col_local] = o;
        else out[(long long)(first + t0 + t) * out_row_stride + (long long)head * vdim + col] = o;
      }
    }
    if (norm.weight != nullptr) {
      __syncthreads();
      const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
      for (int t = warp; t < nt; t += n_warps) {
        const float* o_s = v_s + t * cols;
        float ss = 0.f;
        for (int c = lane; c < vdim; c += 32) ss = fmaf(o_s[c], o_s[c], ss);
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)vdim + norm.eps);
        const long long row = first + t0 + t;
        const T* g = proj + row * row_stride + norm.g_off + (long long)head * vdim;
        T* dst = reinterpret_cast<T*>(norm.mixed) + row * norm.mixed_row_stride + (long long)head * vdim;
        for (int c = lane; c < vdim; c += 32) {
          const float gate = to_float(g[c]);
          dst[c] = from_float<T>(o_s[c] * inv * norm.weight[c] * (gate / (1.f + expf(-gate))));
        }
      }
    }
  }
  if (owns) {
#pragma unroll
    for (int i = 0; i < DPT; ++i)
      if (d0 + i < dim) s_base[(long long)(d0 + i) * vdim + col] = s[i];
  }
}

// lanes a value channel is spread over
static inline int gla_split(int dim) { return dim <= 128 ? 4 : 8; }
static inline bool gla_holds_head(int dim, int vdim) { return gla_split(dim) * vdim <= 512; }

template <typename T>
static int launch_gla_scan(const T* proj, long long row_stride, int q_off, int k_off, int v_off, float q_scale, const float* dt,
                           float log_scale, float* state, const int* slots, const int* seq_start, float* out,
                           long long out_row_stride, int n_seqs, int n_heads, int dim, int vdim, const GlaNorm& norm,
                           cudaStream_t stream) {
  const int split = gla_split(dim);
  int cols = vdim;
  if (!gla_holds_head(dim, vdim)) cols = 512 / split;
  else if (norm.weight == nullptr && cols > 64) cols = 64;        // (more blocks where nothing asks for a whole head)
  const int threads = (split * cols + 31) / 32 * 32;
  const dim3 grid((vdim + cols - 1) / cols, n_heads, n_seqs), block(threads);
  const size_t smem = (size_t)GS_TOKENS * (3 * dim + cols) * sizeof(float);
#define BT_GS(DPT, SPLIT)                                                                                              \
  do {                                                                                                                 \
    auto kernel = gla_scan_kernel<T, DPT, SPLIT>;                                                                      \
    if (smem > 48 * 1024)                                                                                              \
      BT_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) == cudaSuccess,    \
               "gla_scan: cannot reserve %zu bytes of shared memory", smem);                                           \
    BT_PDL_OK("gla_scan", launch_pdl(kernel, grid, block, smem, stream, 1, proj, row_stride, q_off, k_off, v_off, q_scale, \
                                     dt, log_scale, state, slots, seq_start, out, out_row_stride, n_heads, dim, vdim, cols, \
                                     norm));                                                                           \
  } while (0)
  if (dim <= 32) BT_GS(8, 4);
  else if (dim <= 64) BT_GS(16, 4);
  else if (dim <= 128) BT_GS(32, 4);
  else BT_GS(32, 8);
#undef BT_GS
  return 0;
}

// ---- long runs of new tokens: the same recurrence by chunks ------------------------------------------------------
//
// Let b_t be the sum of the log decays up to token t since the chunk's first token (a number per key channel, falling).
// Unrolled over a chunk that starts from S_in,
//
//     o_t   = (q_t e^{b_t})^T S_in + sum_{s <= t} (sum_d q_t[d] k_s[d] e^{b_t[d] - b_s[d]}) v_s
//     S_out = diag(e^{b_end}) S_in + sum_s (k_s e^{b_end - b_s}) v_s^T
//
// e^{-b_s} alone may overflow, so no weight is formed as a quotient: the chunk's 64 tokens lie in 16 groups of four, B_g is
// b at the start of group g, and a weight between groups is the product of three factors that are each at most one,
// e^{b_t - B_g(t)} (kept with q), e^{B_g(t) - B_(g(s)+1)} (formed per pair of groups and channel) and e^{B_(g(s)+1) - b_s}
// (kept with k); inside a group the weights are products of one to three decays.  gla_chunk_kernel forms, per chunk, the
// sums over s, the chunk's own contribution to the state, e^{b_end}, and q_t e^{b_t}; gla_prefix_kernel walks a sequence's
// chunks; gla_carry_kernel adds the incoming state's part.  All 32-bit multiply-adds.

constexpr int GC = 64;     // tokens a chunk
constexpr int GCP = 68;    // row length of the transposed tiles ([channel][token])
constexpr int GG = GC / 4; // groups of four tokens

// grid (chunks, heads * column blocks, sequences); 256 threads; a block owns 64 value channels.
template <typename T>
__global__ void __launch_bounds__(256)
gla_chunk_kernel(const T* __restrict__ proj, long long row_stride, int q_off, int k_off, int v_off, float q_scale,
                 const float* __restrict__ dt, float log_scale, const int* __restrict__ seq_start, float* __restrict__ out,
                 long long out_row_stride, float* __restrict__ states, float* __restrict__ ends, float* __restrict__ aged_q,
                 int max_chunks, int n_heads, int dim, int vdim, int col_blocks) {
  extern __shared__ __align__(16) float sm[];
  float* q_t = sm;                       // [dim][GCP]   q_t e^{b_t - B_g(t)}
  float* k_t = q_t + dim * GCP;          // [dim][GCP]   k_s e^{B_(g(s)+1) - b_s}; then k_s e^{b_end - b_s}
  float* v_s = k_t + dim * GCP;          // [GC][64]
  float* a_t = v_s + GC * 64;            // [GC][GCP]    a_t[s][t]: token t's weight on token s
  float* bs = a_t + GC * GCP;            // [GG + 1][dim]  B_0 .. B_16
  pdl_trigger();
  pdl_wait();
  const int chunk = blockIdx.x, seq = blockIdx.z;
  const int head = blockIdx.y / col_blocks, col_block = blockIdx.y - head * col_blocks, col0 = col_block * 64;
  const int first = seq_start[seq], n_new = seq_start[seq + 1] - first;
  if (chunk * GC >= n_new) return;
  const int len = min(GC, n_new - chunk * GC);
  const long long row0 = first + (long long)chunk * GC;
  const int tid = threadIdx.x, ty = tid >> 4, tx = tid & 15, warp = tid >> 5, lane = tid & 31;
  for (int i = tid; i < GC * 64; i += 256) {
    const int t = i >> 6, c = i & 63;
    v_s[i] = (t < len && col0 + c < vdim)
                 ? to_float(proj[(row0 + t) * row_stride + v_off + (long long)head * vdim + col0 + c]) : 0.f;
  }
  // a warp takes two groups, a lane a channel: the group's q, k and decays, and the weights inside the group
  for (int g = warp * 2; g < warp * 2 + 2; ++g) {
    float w00 = 0.f, w11 = 0.f, w22 = 0.f, w33 = 0.f, w10 = 0.f, w21 = 0.f, w32 = 0.f, w20 = 0.f, w31 = 0.f, w30 = 0.f;
    for (int d = lane; d < dim; d += 32) {
      float q[4], k[4], la[4], a[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = 4 * g + i;
        q[i] = k[i] = la[i] = 0.f;
        if (t < len) {
          const T* src = proj + (row0 + t) * row_stride + (long long)head * dim + d;
          q[i] = to_float(src[q_off]) * q_scale;
          k[i] = to_float(src[k_off]);
          la[i] = dt[((row0 + t) * n_heads + head) * dim + d] * log_scale;
        }
        a[i] = gla_exp<T>(la[i]);
      }
      bs[(g + 1) * dim + d] = (la[0] + la[1]) + (la[2] + la[3]);
      const float a12 = a[1] * a[2], a23 = a[2] * a[3], a123 = a12 * a[3];
      w00 = fmaf(q[0], k[0], w00);
      w11 = fmaf(q[1], k[1], w11);
      w22 = fmaf(q[2], k[2], w22);
      w33 = fmaf(q[3], k[3], w33);
      w10 = fmaf(q[1], k[0] * a[1], w10);
      w21 = fmaf(q[2], k[1] * a[2], w21);
      w32 = fmaf(q[3], k[2] * a[3], w32);
      w20 = fmaf(q[2], k[0] * a12, w20);
      w31 = fmaf(q[3], k[1] * a23, w31);
      w30 = fmaf(q[3], k[0] * a123, w30);
      const float p1 = a[0] * a[1], p2 = p1 * a[2], p3 = p2 * a[3];
      *reinterpret_cast<float4*>(q_t + d * GCP + 4 * g) = make_float4(q[0] * a[0], q[1] * p1, q[2] * p2, q[3] * p3);
      *reinterpret_cast<float4*>(k_t + d * GCP + 4 * g) = make_float4(k[0] * a123, k[1] * a23, k[2] * a[3], k[3]);
    }
    w00 = warp_sum(w00); w11 = warp_sum(w11); w22 = warp_sum(w22); w33 = warp_sum(w33); w10 = warp_sum(w10);
    w21 = warp_sum(w21); w32 = warp_sum(w32); w20 = warp_sum(w20); w31 = warp_sum(w31); w30 = warp_sum(w30);
    if (lane == 0) {
      float* cell = a_t + 4 * g * GCP + 4 * g;      // [s][t]
      *reinterpret_cast<float4*>(cell) = make_float4(w00, w10, w20, w30);
      *reinterpret_cast<float4*>(cell + GCP) = make_float4(0.f, w11, w21, w31);
      *reinterpret_cast<float4*>(cell + 2 * GCP) = make_float4(0.f, 0.f, w22, w32);
      *reinterpret_cast<float4*>(cell + 3 * GCP) = make_float4(0.f, 0.f, 0.f, w33);
    }
  }
  __syncthreads();
  for (int d = tid; d < dim; d += 256) {
    float sum = 0.f;
    bs[d] = 0.f;
    for (int g = 1; g <= GG; ++g) {
      sum += bs[g * dim + d];
      bs[g * dim + d] = sum;
    }
    if (col_block == 0) ends[(((long long)seq * max_chunks + chunk) * n_heads + head) * dim + d] = gla_exp<T>(sum);
  }
  __syncthreads();
  if (col_block == 0)
    for (int i = tid; i < len * dim; i += 256) {
      const int t = i / dim, d = i - t * dim;
      aged_q[((row0 + t) * n_heads + head) * dim + d] = q_t[d * GCP + t] * gla_exp<T>(bs[(t >> 2) * dim + d]);
    }
  // weights between groups: 120 pairs (later group gt, earlier group gs), each shared by two threads with half of the channels
  {
    const int pair = tid & 127, half = tid >> 7;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    int gt = 1;
    while (gt < GG - 1 && (gt + 1) * gt / 2 <= pair) ++gt;
    const int gs = pair - gt * (gt - 1) / 2;
    const bool live = pair < GG * (GG - 1) / 2 && 4 * gt < len;
    float* cell = a_t + 4 * gs * GCP + 4 * gt;
    if (live) {
      const int d_mid = (dim + 1) / 2, d_end = half ? dim : d_mid;
      const float* bt_ = bs + gt * dim;
      const float* bq = bs + (gs + 1) * dim;
      for (int d = half ? d_mid : 0; d < d_end; ++d) {
        const float f = gla_exp<T>(bt_[d] - bq[d]);
        const float4 qv = *reinterpret_cast<const float4*>(q_t + d * GCP + gt * 4);
        const float4 kv = *reinterpret_cast<const float4*>(k_t + d * GCP + gs * 4);
        const float qa[4] = {qv.x, qv.y, qv.z, qv.w}, ka[4] = {kv.x * f, kv.y * f, kv.z * f, kv.w * f};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(qa[i], ka[j], acc[i][j]);
      }
      if (half)
#pragma unroll
        for (int j = 0; j < 4; ++j)
          *reinterpret_cast<float4*>(cell + j * GCP) = make_float4(acc[0][j], acc[1][j], acc[2][j], acc[3][j]);
    }
    __syncthreads();
    if (live && !half) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float4* at = reinterpret_cast<float4*>(cell + j * GCP);
        const float4 o = *at;
        *at = make_float4(acc[0][j] + o.x, acc[1][j] + o.y, acc[2][j] + o.z, acc[3][j] + o.w);
      }
    }
  }
  __syncthreads();
  // k_s e^{b_end - b_s}
  for (int i = tid; i < GG * dim; i += 256) {
    const int g = i / dim, d = i - g * dim;
    const float f = gla_exp<T>(bs[GG * dim + d] - bs[(g + 1) * dim + d]);
    float4* at = reinterpret_cast<float4*>(k_t + d * GCP + 4 * g);
    const float4 kv = *at;
    *at = make_float4(kv.x * f, kv.y * f, kv.z * f, kv.w * f);
  }
  // the part of o_t that needs no earlier chunk: tokens 4 ty .., channels 4 tx ..
  {
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    const int s_end = ty * 4 < len ? min(len, ty * 4 + 4) : 0;
    for (int sx = 0; sx < s_end; ++sx) {
      const float4 av = *reinterpret_cast<const float4*>(a_t + sx * GCP + ty * 4);
      const float4 vv = *reinterpret_cast<const float4*>(v_s + sx * 64 + tx * 4);
      const float aa[4] = {av.x, av.y, av.z, av.w}, va[4] = {vv.x, vv.y, vv.z, vv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(aa[i], va[j], acc[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = ty * 4 + i;
      if (t >= len) break;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int c = col0 + tx * 4 + j;
        if (c < vdim) out[(row0 + t) * out_row_stride + (long long)head * vdim + c] = acc[i][j];
      }
    }
  }
  __syncthreads();
  // the chunk's contribution to the state, key channels 4 ty .. (+ 64, ...)
  float* dst = states + ((((long long)seq * max_chunks + chunk) * n_heads + head) * dim) * vdim;
  for (int i0 = ty * 4; i0 < dim; i0 += 64) {
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int sx = 0; sx < len; ++sx) {
      const float4 vv = *reinterpret_cast<const float4*>(v_s + sx * 64 + tx * 4);
      const float va[4] = {vv.x, vv.y, vv.z, vv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float kv = i0 + i < dim ? k_t[(i0 + i) * GCP + sx] : 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(kv, va[j], acc[i][j]);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int c = col0 + tx * 4 + j;
        if (i0 + i < dim && c < vdim) dst[(long long)(i0 + i) * vdim + c] = acc[i][j];
      }
  }
}

// One thread per (sequence, head, state element): walks the sequence's chunks in order; leaves in states[chunk] the state
// that chunk STARTS from and in `state` the state after the last one.  Four chunks are asked for at a time.
__global__ void __launch_bounds__(256)
gla_prefix_kernel(float* states, const float* __restrict__ ends, float* __restrict__ state, const int* __restrict__ slots,
                  const int* __restrict__ seq_start, int max_chunks, int n_heads, int dim, int vdim) {
  pdl_trigger();
  pdl_wait();
  const int seq = blockIdx.z, head = blockIdx.y;
  const int e = blockIdx.x * 256 + threadIdx.x;
  if (e >= dim * vdim) return;
  const int n_new = seq_start[seq + 1] - seq_start[seq];
  const int n_chunks = (n_new + GC - 1) / GC;
  float* st = state + (((long long)slots[seq] * n_heads + head) * dim) * vdim + e;
  const long long stride = (long long)n_heads * dim * vdim, end_stride = (long long)n_heads * dim;
  float* cell = states + (((long long)seq * max_chunks) * n_heads + head) * (long long)dim * vdim + e;
  const float* end = ends + ((long long)seq * max_chunks * n_heads + head) * dim + e / vdim;
  float s = *st;
  for (int c = 0; c < n_chunks; c += 4) {
    float kv[4], decay[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      kv[u] = c + u < n_chunks ? __ldcg(cell + (c + u) * stride) : 0.f;
      decay[u] = c + u < n_chunks ? end[(c + u) * end_stride] : 0.f;
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (c + u < n_chunks) {
        cell[(c + u) * stride] = s;
        s = fmaf(decay[u], s, kv[u]);
      }
    }
  }
  *st = s;
}

// out[t] += (q_t e^{b_t})^T S_in for the tokens of a chunk; grid and blocks as gla_chunk_kernel.
__global__ void __launch_bounds__(256)
gla_carry_kernel(const float* __restrict__ aged_q, const int* __restrict__ seq_start, float* __restrict__ out,
                 long long out_row_stride, const float* __restrict__ states, int max_chunks, int n_heads, int dim, int vdim,
                 int col_blocks) {
  extern __shared__ __align__(16) float sm[];
  float* q_t = sm;                 // [dim][GCP]
  float* s_s = q_t + dim * GCP;    // [dim][64]
  pdl_trigger();
  pdl_wait();
  const int chunk = blockIdx.x, seq = blockIdx.z;
  const int head = blockIdx.y / col_blocks, col0 = (blockIdx.y - head * col_blocks) * 64;
  const int first = seq_start[seq], n_new = seq_start[seq + 1] - first;
  if (chunk * GC >= n_new) return;
  const int len = min(GC, n_new - chunk * GC);
  const long long row0 = first + (long long)chunk * GC;
  const int tid = threadIdx.x, ty = tid >> 4, tx = tid & 15;
  for (int i = tid; i < GC * dim; i += 256) {
    const int t = i / dim, d = i - t * dim;
    q_t[d * GCP + t] = t < len ? aged_q[((row0 + t) * n_heads + head) * dim + d] : 0.f;
  }
  const float* src = states + ((((long long)seq * max_chunks + chunk) * n_heads + head) * dim) * vdim + col0;
  for (int i = tid; i < dim * 64; i += 256) {
    const int d = i >> 6, c = i & 63;
    s_s[i] = col0 + c < vdim ? src[(long long)d * vdim + c] : 0.f;
  }
  __syncthreads();
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int d = 0; d < dim; ++d) {
    const float4 qv = *reinterpret_cast<const float4*>(q_t + d * GCP + ty * 4);
    const float4 sv = *reinterpret_cast<const float4*>(s_s + d * 64 + tx * 4);
    const float qa[4] = {qv.x, qv.y, qv.z, qv.w}, sa[4] = {sv.x, sv.y, sv.z, sv.w};
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(qa[i], sa[j], acc[i][j]);
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = ty * 4 + i;
    if (t >= len) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = col0 + tx * 4 + j;
      if (c < vdim) out[(row0 + t) * out_row_stride + (long long)head * vdim + c] += acc[i][j];
    }
  }
}

// Scratch of the chunked form: [states | ends | aged_q].
static inline long long gla_state_floats(int n_seqs, int max_new, int n_heads, int dim, int vdim) {
  return (long long)n_seqs * ((max_new + GC - 1) / GC) * n_heads * dim * vdim;
}
static inline long long gla_end_floats(int n_seqs, int max_new, int n_heads, int dim) {
  return (long long)n_seqs * ((max_new + GC - 1) / GC) * n_heads * dim;
}

template <typename T>
static int launch_gla_chunked(const T* proj, long long row_stride, int q_off, int k_off, int v_off, float q_scale,
                              const float* dt, float log_scale, float* state, const int* slots, const int* seq_start,
                              float* out, long long out_row_stride, float* scratch, int max_new, int n_seqs, int n_heads,
                              int dim, int vdim, cudaStream_t stream) {
  const int col_blocks = (vdim + 63) / 64, max_chunks = (max_new + GC - 1) / GC;
  BT_CHECK((long long)n_heads * col_blocks <= 65535, "gla: %d heads x %d column blocks are too many", n_heads, col_blocks);
  const dim3 grid(max_chunks, n_heads * col_blocks, n_seqs), block(256);
  const size_t smem_a = ((size_t)2 * dim * GCP + (size_t)GC * 64 + (size_t)GC * GCP + (size_t)(GG + 1) * dim) * sizeof(float);
  const size_t smem_c = ((size_t)dim * GCP + (size_t)dim * 64) * sizeof(float);
  auto chunk_kernel = gla_chunk_kernel<T>;
  if (smem_a > 48 * 1024)
    BT_CHECK(cudaFuncSetAttribute(chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_a) == cudaSuccess,
             "gla: cannot reserve %zu bytes of shared memory", smem_a);
  if (smem_c > 48 * 1024)
    BT_CHECK(cudaFuncSetAttribute(gla_carry_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_c) == cudaSuccess,
             "gla: cannot reserve %zu bytes of shared memory", smem_c);
  float* states = scratch;
  float* ends = states + gla_state_floats(n_seqs, max_new, n_heads, dim, vdim);
  float* aged_q = ends + gla_end_floats(n_seqs, max_new, n_heads, dim);
  BT_PDL_OK("gla_chunk", launch_pdl(chunk_kernel, grid, block, smem_a, stream, 1, proj, row_stride, q_off, k_off, v_off, q_scale,
                                    dt, log_scale, seq_start, out, out_row_stride, states, ends, aged_q, max_chunks, n_heads,
                                    dim, vdim, col_blocks));
  BT_PDL_OK("gla_prefix", launch_pdl(gla_prefix_kernel, dim3((dim * vdim + 255) / 256, n_heads, n_seqs), block, 0, stream, 1,
                                     states, (const float*)ends, state, slots, seq_start, max_chunks, n_heads, dim, vdim));
  BT_PDL_OK("gla_carry", launch_pdl(gla_carry_kernel, grid, block, smem_c, stream, 1, (const float*)aged_q, seq_start, out,
                                    out_row_stride, (const float*)states, max_chunks, n_heads, dim, vdim, col_blocks));
  return 0;
}

}  // namespace bt

// Whether the token-by-token kernel holds a whole head of this size in one block (and can norm and gate it).
extern "C" int bt_gla_scan_fuses(int dim, int vdim) { return bt::gla_holds_head(dim, vdim) ? 1 : 0; }

// norm_weight (null: none): see GlaNorm; the read-out then goes to `mixed` (rows of proj's type) and `out` is not written.
extern "C" int bt_gla_scan(const void* proj, long long row_stride, int q_off, int k_off, int v_off, float q_scale,
                           const float* dt, float log_scale, float* state, const int* slots, const int* seq_start, float* out,
                           long long out_row_stride, int n_seqs, int n_heads, int dim, int vdim, const float* norm_weight,
                           float eps, int g_off, void* mixed, long long mixed_row_stride, int dtype, cudaStream_t stream) {
  using namespace bt;
  BT_CHECK(n_heads > 0 && dim > 0 && dim <= 256 && vdim > 0 && n_seqs >= 0 && n_seqs <= 65535 && n_heads <= 65535,
           "gla_scan: bad sizes seqs=%d heads=%d dim=%d vdim=%d", n_seqs, n_heads, dim, vdim);
  BT_CHECK(norm_weight == nullptr || gla_holds_head(dim, vdim), "gla_scan: no block holds a head of %d x %d", dim, vdim);
  BT_CHECK(norm_weight != nullptr ? mixed != nullptr : out != nullptr, "gla_scan: nowhere to leave the result");
  if (n_seqs == 0) return 0;
  const GlaNorm norm{norm_weight, eps, g_off, mixed, mixed_row_stride};
  if (dtype == kF32)
    return launch_gla_scan<float>((const float*)proj, row_stride, q_off, k_off, v_off, q_scale, dt, log_scale, state, slots,
                                  seq_start, out, out_row_stride, n_seqs, n_heads, dim, vdim, norm, stream);
  if (dtype == kBF16)
    return launch_gla_scan<__nv_bfloat16>((const __nv_bfloat16*)proj, row_stride, q_off, k_off, v_off, q_scale, dt, log_scale,
                                          state, slots, seq_start, out, out_row_stride, n_seqs, n_heads, dim, vdim, norm, stream);
  return fail("gla_scan: unknown dtype %d", dtype);
}

// The same results as bt_gla_scan (beyond rounding), the chunks of a run worked side by side; `out` [tokens][heads vdim].
// scratch: (n_seqs * chunks of max_new) * n_heads * dim * (vdim + 1) + n_tokens * n_heads * dim floats.
extern "C" int bt_gla_chunked(const void* proj, long long row_stride, int q_off, int k_off, int v_off, float q_scale,
                              const float* dt, float log_scale, float* state, const int* slots, const int* seq_start,
                              float* out, long long out_row_stride, float* scratch, int max_new, int n_seqs, int n_heads,
                              int dim, int vdim, int dtype, cudaStream_t stream) {
  using namespace bt;
  BT_CHECK(n_heads > 0 && dim > 0 && dim <= 256 && vdim > 0 && n_seqs >= 0 && n_seqs <= 65535 && max_new > 0 && scratch,
           "gla_chunked: bad sizes seqs=%d heads=%d dim=%d vdim=%d max_new=%d", n_seqs, n_heads, dim, vdim, max_new);
  if (n_seqs == 0) return 0;
  if (dtype == kF32)
    return launch_gla_chunked<float>((const float*)proj, row_stride, q_off, k_off, v_off, q_scale, dt, log_scale, state, slots,
                                     seq_start, out, out_row_stride, scratch, max_new, n_seqs, n_heads, dim, vdim, stream);
  if (dtype == kBF16)
    return launch_gla_chunked<__nv_bfloat16>((const __nv_bfloat16*)proj, row_stride, q_off, k_off, v_off, q_scale, dt, log_scale,
                                             state, slots, seq_start, out, out_row_stride, scratch, max_new, n_seqs, n_heads, dim,
                                             vdim, stream);
  return fail("gla_chunked: unknown dtype %d", dtype);
}
