// Recurrences of a matrix state per head under one decay per head and token: the gated delta rule, the
// state-space (Mamba-2) update and the update under a fixed decay per head (lightning attention), with the short
// convolutions in front of them and the gated norms behind.
//
// Per head, with a state S [dim, vdim] (float32, zero at a sequence's start, kept per slot), a log decay l_t and a
// factor b_t (both from per-head pre-activations):
//
//   delta rule     S' = e^l S;  u = b (v - S'^T k);  S = S' + k u^T;  o = S^T q       b = sigmoid(.),
//                  q and k unit vectors per head, q times a scale                     l = -e^A softplus(. + bias)
//   state space    S' = e^l S;  S = S' + b k v^T;    o = S^T q + D v                  b = softplus(. + bias), l = -e^A b
//                  (k: the input matrix B, q: the read-out C, v: the inner input x)
//   fixed decay    the state-space update with b = 1 and one log decay per head, the same for every token
//
// q and k belong to groups of heads (head h uses group h / (heads / groups)).  In front, every channel of q, k and v
// goes through a short convolution along the sequence (optionally with a bias) and SiLU.  All of it float32.
//
// Per-slot state, float32: [heads][dim][vdim] the matrices, then (taps > 1) a ring of the convolutions' inputs,
// [taps][channels] with channels = q, k, v: the input of position p lies in row p % taps.  A step of one token reads the
// rows of the taps - 1 positions before it and writes its own, which none of its readers asks for, so the blocks of
// such a step need no order among themselves: convolution, gates and recurrence are one launch.
#include "common.cuh"

#define GS_MAX_TAPS 16
#define GS_WARPS 8
#define GS_THREADS (GS_WARPS * 32)

__device__ __forceinline__ float gs_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float gs_silu(float z) { return z / (1.0f + expf(-z)); }

// What the kernels need to find things: the rows of the projection (element type T) with the channels of q, k, v at
// their offsets, the float32 pre-activations of the heads' gates, and the step.
struct GatedStateArgs {
  const void* proj;
  const float* gate;          // [tokens, gate_stride]: log decays' (or step sizes') pre-activations at a_off, delta: b's at b_off
  const float* log_decay;     // [heads]: fixed log decays (no gates are read then), or null
  const float* conv_w;        // [taps][channels], or null: no convolution (taps = 1)
  const float* conv_b;        // [channels] or null
  const float* dt_bias;       // [heads]
  const float* a_log;         // [heads]
  const float* d;             // [heads] or null
  float* state;
  const int* tok_seq;
  const int* seq_start;
  const int* seq_pos0;
  const int* slots;
  size_t state_stride;
  float q_scale;
  int stride, gate_stride, q_off, k_off, v_off, a_off, b_off, groups, heads, dim, vdim, taps, n_seqs, n_tokens;
  __device__ __forceinline__ int n_qk() const { return groups * dim; }
  __device__ __forceinline__ int n_ch() const { return 2 * groups * dim + heads * vdim; }
  __device__ __forceinline__ int column(int c) const {
    const int n = groups * dim;
    return c < n ? q_off + c : (c < 2 * n ? k_off + c - n : v_off + c - 2 * n);
  }
  __device__ __forceinline__ const float* ring(int s) const {
    return state + (size_t)slots[s] * state_stride + (size_t)heads * dim * vdim;
  }
};

// (log decay, factor) of a head at a token
template <bool DELTA>
__device__ __forceinline__ float2 gs_gates(const GatedStateArgs& a, int t, int h) {
  if (!DELTA && a.log_decay) return make_float2(a.log_decay[h], 1.0f);
  const float* g = a.gate + (size_t)t * a.gate_stride;
  const float dt = gs_softplus(g[a.a_off + h] + a.dt_bias[h]);
  const float beta = DELTA ? 1.0f / (1.0f + expf(-g[a.b_off + h])) : dt;
  return make_float2(-expf(a.a_log[h]) * dt, beta);
}

// ---- runs of tokens: everything in front of the recurrence ------------------------------------------
template <typename T, int V>
__device__ __forceinline__ void gs_load(const T* p, float* o);
template <>
__device__ __forceinline__ void gs_load<float, 4>(const float* p, float* o) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w;
}
template <>
__device__ __forceinline__ void gs_load<__nv_bfloat16, 4>(const __nv_bfloat16* p, float* o) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  o[0] = a.x; o[1] = a.y; o[2] = b.x; o[3] = b.y;
}
template <>
__device__ __forceinline__ void gs_load<float, 1>(const float* p, float* o) { o[0] = *p; }
template <>
__device__ __forceinline__ void gs_load<__nv_bfloat16, 1>(const __nv_bfloat16* p, float* o) { o[0] = __bfloat162float(*p); }

// One block per token: convolution and SiLU of every channel (q and k wait in shared memory for their unit norms in
// the delta rule), log decays and factors.  qn, kn [T, groups * dim], vc [T, heads * vdim], lb [T, heads, 2].
template <typename T, int V, bool DELTA>
__global__ void gated_state_prepare_kernel(const GatedStateArgs a, float* __restrict__ qn, float* __restrict__ kn,
                                           float* __restrict__ vc, float* __restrict__ lb) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float ch[];  // delta: the q and k channels after convolution and SiLU
  const int t = blockIdx.x, s = a.tok_seq[t], start = a.seq_start[s], r = t - start, pos = a.seq_pos0[s] + r;
  const int n_qk = a.n_qk(), n_ch = a.n_ch();
  const T* proj = (const T*)a.proj;
  const float* ring = a.ring(s);
  for (int c = threadIdx.x * V; c < n_ch; c += blockDim.x * V) {
    const int col = a.column(c);
    float acc[V];
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] = 0.f;
    if (a.conv_b) gs_load<float, V>(a.conv_b + c, acc);
    for (int j = 0; j < a.taps; ++j) {
      const int back = a.taps - 1 - j;  // how many positions before this token the tap looks
      if (back > pos) continue;         // no such position
      float x[V], w[V];
      if (a.conv_w) {
        gs_load<float, V>(a.conv_w + (size_t)j * n_ch + c, w);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) w[e] = 1.0f;
      }
      if (r - back >= 0) gs_load<T, V>(proj + (size_t)(t - back) * a.stride + col, x);
      else gs_load<float, V>(ring + (size_t)((pos - back) % a.taps) * n_ch + c, x);
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = fmaf(w[e], x[e], acc[e]);
    }
    float* dst;
    if (c >= 2 * n_qk) dst = vc + (size_t)t * (n_ch - 2 * n_qk) + c - 2 * n_qk;
    else if (DELTA) dst = ch + c;
    else dst = c < n_qk ? qn + (size_t)t * n_qk + c : kn + (size_t)t * n_qk + c - n_qk;
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] = gs_silu(acc[e]);
    if (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(acc[0], acc[1 % V], acc[2 % V], acc[3 % V]);
    else dst[0] = acc[0];
  }
  for (int h = threadIdx.x; h < a.heads; h += blockDim.x) {
    const float2 g = gs_gates<DELTA>(a, t, h);
    lb[((size_t)t * a.heads + h) * 2] = g.x;
    lb[((size_t)t * a.heads + h) * 2 + 1] = g.y;
  }
  if (!DELTA) return;
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  for (int item = warp; item < 2 * a.groups; item += n_warps) {  // q heads, then k heads
    const float* v = ch + (size_t)item * a.dim;
    float ss = 0.f;
    for (int i = lane; i < a.dim; i += 32) ss = fmaf(v[i], v[i], ss);
    ss = warp_sum(ss);
    const bool is_q = item < a.groups;
    const float scale = (1.0f / sqrtf(ss + 1e-6f)) * (is_q ? a.q_scale : 1.0f);
    float* dst = (is_q ? qn : kn) + (size_t)t * n_qk + (size_t)(is_q ? item : item - a.groups) * a.dim;
    for (int i = lane; i < a.dim; i += 32) dst[i] = v[i] * scale;
  }
}

// What later tokens ask for of a run's inputs, into the ring: the block of (head, column tile) keeps its value channels, the
// first block of a group's first head the group's q and k channels.  Runs after everybody has read the ring.
template <typename T>
__device__ __forceinline__ void gs_keep_inputs(const GatedStateArgs& a, int s, int h, int col0, int cols, bool with_qk) {
  if (a.taps < 2) return;
  const int start = a.seq_start[s], n = a.seq_start[s + 1] - start, pos0 = a.seq_pos0[s];
  const int n_qk = a.n_qk(), n_ch = a.n_ch();
  float* ring = const_cast<float*>(a.ring(s));
  const int per_group = a.heads / a.groups, g = h / per_group;
  const int n_own = cols + (with_qk ? 2 * a.dim : 0);
  for (int r = max(0, n - (a.taps - 1)); r < n; ++r) {
    float* row = ring + (size_t)((pos0 + r) % a.taps) * n_ch;
    const T* src = (const T*)a.proj + (size_t)(start + r) * a.stride;
    for (int i = threadIdx.x; i < n_own; i += blockDim.x) {
      const int j = i - cols;
      const int c = j < 0 ? 2 * n_qk + h * a.vdim + col0 + i : (j < a.dim ? g * a.dim + j : n_qk + g * a.dim + j - a.dim);
      row[c] = to_f32<T>(src[a.column(c)]);
    }
  }
}

// The recurrence, token by token.  A block of eight warps per (sequence, head, 32 value columns): a lane holds its
// column of S in registers, a warp an eighth of the rows (RW each, a multiple of 4); the tokens' q and k rows pass
// through shared memory four tokens deep (rows past dim are zeros), and one barrier per token is enough.  What a token
// needs from memory is asked for three tokens ahead.  o = (e^l S)^T q + (k . q) u, so both read-outs of the decayed
// state are taken in one pass over the rows.
template <typename T, int RW, bool DELTA>
__global__ void __launch_bounds__(GS_THREADS) gated_state_kernel(const GatedStateArgs a, const float* __restrict__ qn,
                                                                 const float* __restrict__ kn, const float* __restrict__ vc,
                                                                 const float* __restrict__ lb, int col_tiles,
                                                                 float* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int ROWS = GS_WARPS * RW;                  // rows of the padded state, >= dim
  __shared__ __align__(16) float in[4][2][ROWS];       // [token % 4][q, k][row]
  __shared__ float red[2][GS_WARPS][65];               // the warps' partial read-outs and k . q
  const int heads = a.heads, dim = a.dim, vdim = a.vdim;
  const int tile = blockIdx.x % col_tiles, h = (blockIdx.x / col_tiles) % heads, s = blockIdx.x / (col_tiles * heads);
  const int per_group = heads / a.groups, g = h / per_group;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int col = tile * 32 + lane;
  const bool live = col < vdim;
  const int row0 = warp * RW;
  const int start = a.seq_start[s], n = a.seq_start[s + 1] - start;
  float* S_g = a.state + (size_t)a.slots[s] * a.state_stride + (size_t)h * dim * vdim;
  float S[RW];
#pragma unroll
  for (int i = 0; i < RW; ++i) S[i] = (live && row0 + i < dim) ? S_g[(size_t)(row0 + i) * vdim + col] : 0.f;
  const int n_qk = a.n_qk();
  const float skip = a.d ? a.d[h] : 0.f;
  const int my_row = threadIdx.x;  // a thread fetches at most one row of a token: ROWS <= GS_THREADS
  const bool fetches = my_row < ROWS, in_dim = my_row < dim;
  auto fetch = [&](int tok, float& q, float& k) {
    const size_t at = (size_t)(start + tok) * n_qk + (size_t)g * dim + my_row;
    q = in_dim ? qn[at] : 0.f;
    k = in_dim ? kn[at] : 0.f;
  };
  auto put = [&](int buf, float q, float k) {
    if (fetches) { in[buf][0][my_row] = q; in[buf][1][my_row] = k; }
  };
  float nq = 0.f, nk = 0.f;  // the rows of token tok + 2
  {
    float q, k;
    if (n > 0 && fetches) { fetch(0, q, k); put(0, q, k); }
    if (n > 1 && fetches) { fetch(1, q, k); put(1, q, k); }
    if (n > 2 && fetches) fetch(2, nq, nk);
  }
  __syncthreads();
  auto v_of = [&](int tok) { return live ? vc[(size_t)(start + tok) * heads * vdim + (size_t)h * vdim + col] : 0.f; };
  auto g_of = [&](int tok) { return *reinterpret_cast<const float2*>(lb + ((size_t)(start + tok) * heads + h) * 2); };
  const float2 zero2 = make_float2(0.f, 0.f);
  float v0 = n > 0 ? v_of(0) : 0.f, v1 = n > 1 ? v_of(1) : 0.f;
  float2 g0 = n > 0 ? g_of(0) : zero2, g1 = n > 1 ? g_of(1) : zero2;
  for (int tok = 0; tok < n; ++tok) {
    const int buf = tok & 3;
    const float v = v0, bt = g0.y, decay = expf(g0.x);
    v0 = v1; g0 = g1;
    if (tok + 2 < n) {
      v1 = v_of(tok + 2);
      g1 = g_of(tok + 2);
      put((tok + 2) & 3, nq, nk);  // the buffer of token tok - 2: every warp has left it (the barrier of tok - 1)
    }
    if (tok + 3 < n && fetches) fetch(tok + 3, nq, nk);
    float pk = 0.f, pq = 0.f, kq = 0.f;
    float kreg[RW];
#pragma unroll
    for (int i = 0; i < RW; i += 4) {
      const float4 q4 = *reinterpret_cast<const float4*>(&in[buf][0][row0 + i]);
      const float4 k4 = *reinterpret_cast<const float4*>(&in[buf][1][row0 + i]);
      const float qs[4] = {q4.x, q4.y, q4.z, q4.w}, ks[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float sd = S[i + e] * decay;
        S[i + e] = sd;
        kreg[i + e] = ks[e];
        if (DELTA) pk = fmaf(sd, ks[e], pk);
        pq = fmaf(sd, qs[e], pq);
        kq = fmaf(ks[e], qs[e], kq);
      }
    }
    float* rd = &red[tok & 1][0][0];
    if (DELTA) rd[warp * 65 + lane] = pk;
    rd[warp * 65 + 32 + lane] = pq;
    if (lane == 0) rd[warp * 65 + 64] = kq;
    __syncthreads();
    float sk = 0.f, sq = 0.f, skq = 0.f;
    if (DELTA) {
#pragma unroll
      for (int w = 0; w < GS_WARPS; ++w) sk += rd[w * 65 + lane];
    }
    const float u = bt * (v - sk);
#pragma unroll
    for (int i = 0; i < RW; ++i) S[i] = fmaf(kreg[i], u, S[i]);
    if (warp == 0 && live) {
#pragma unroll
      for (int w = 0; w < GS_WARPS; ++w) {
        sq += rd[w * 65 + 32 + lane];
        skq += rd[w * 65 + 64];
      }
      out[(size_t)(start + tok) * heads * vdim + (size_t)h * vdim + col] = fmaf(skip, v, fmaf(skq, u, sq));
    }
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < RW; ++i)
      if (row0 + i < dim) S_g[(size_t)(row0 + i) * vdim + col] = S[i];
  }
  gs_keep_inputs<T>(a, s, h, tile * 32, min(32, vdim - tile * 32), tile == 0 && h % per_group == 0);
}

// ---- runs of many tokens: the recurrence chunk by chunk ------------------------------------------------
// Within a chunk of 64 tokens the recurrence is unrolled into sums.  With c_t the sum of the log decays from the chunk's
// first token to t and S0 the state before the chunk,
//
//   o_t = e^{c_t} S0^T q_t + sum_{s <= t} e^{c_t - c_s} (q_t . k_s) u_s,      S_end = e^{c_end} S0 + sum_s e^{c_end - c_s} k_s u_s^T
//
// where u_s = b_s v_s for the state-space update.  In the delta rule u solves a unit lower triangular system,
// (I + A) U = diag(b) (V - diag(e^c) K S0) with A_ts = b_t e^{c_t - c_s} (k_t . k_s) for s < t: its inverse depends on the
// chunk alone.  (I + A)^-1 diag(b) of every chunk and head, and q_t . k_s of every chunk and group, come from a first
// kernel, all chunks at once; a second one carries the state through the chunks with small float32 products.  Every
// exponent is at most zero.  The sums run in another order than token by token: the forms agree to rounding.
#define GC_L 64
#define GC_THREADS 256
#define GC_CHAIN_THREADS 512
#define GC_PLD 68  // padded rows of the chunk's 64 x 64 matrices

__device__ __forceinline__ void gc_copy16(float* smem, const float* gmem, bool valid) {
  const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
  const int n = valid ? 16 : 0;  // zeros where there is nothing to read
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(gmem), "r"(n) : "memory");
}
__device__ __forceinline__ void gc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void gc_wait() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// Which 16-byte pieces of 64 rows of `cols` numbers (a multiple of four) a thread copies: from (row, col) on, always
// (d_row, d_col) further.
struct CopyPlan {
  int row, col, d_row, d_col, per_row;
  __device__ __forceinline__ explicit CopyPlan(int cols) {
    per_row = cols >> 2;
    row = threadIdx.x / per_row;
    col = threadIdx.x - row * per_row;
    d_row = blockDim.x / per_row;
    d_col = blockDim.x - d_row * per_row;
  }
};
// 64 rows of the matrix at src (src_ld apart) to dst (dst_ld apart), zeros past n_valid rows
__device__ __forceinline__ void gc_load_rows(const CopyPlan& p, float* dst, int dst_ld, const float* src, size_t src_ld, int n_valid) {
  for (int r = p.row, c = p.col; r < GC_L;) {
    gc_copy16(dst + r * dst_ld + c * 4, src + (size_t)(r < n_valid ? r : 0) * src_ld + c * 4, r < n_valid);
    r += p.d_row;
    c += p.d_col;
    if (c >= p.per_row) {
      c -= p.per_row;
      ++r;
    }
  }
}

// Sums of the log decays over a chunk's tokens, by one warp: lane holds tokens 2 lane and 2 lane + 1.
__device__ __forceinline__ float2 gc_cumulate(float l0, float l1, int lane) {
  float both = l0 + l1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float up = __shfl_up_sync(0xffffffffu, both, o);
    if (lane >= o) both += up;
  }
  return make_float2(both - l1, both);
}

// One block per (chunk, head) in the delta rule, per (chunk, group) otherwise.  qk [T, groups, 64]: q_t . k_s for the
// tokens s of t's chunk; winv [T, heads, 64]: the rows of (I + A)^-1 diag(b).
template <bool DELTA>
__global__ void __launch_bounds__(GC_THREADS) gated_state_local_kernel(const GatedStateArgs a, const float* __restrict__ qn,
                                                                       const float* __restrict__ kn, const float* __restrict__ lb,
                                                                       const int* __restrict__ tile_seq, const int* __restrict__ tile_row0,
                                                                       float* __restrict__ qk, float* __restrict__ winv) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  const int dim = a.dim, ld = dim + 4;
  float* sK = sm;
  float* sQ = sK + GC_L * ld;
  float* sA = sQ + GC_L * ld;  // [64][GC_PLD]
  __shared__ float sc[GC_L], sb[GC_L];
  const int h = DELTA ? blockIdx.y : 0, per_group = a.heads / a.groups, g = DELTA ? h / per_group : blockIdx.y;
  const int s = tile_seq[blockIdx.x], row0 = tile_row0[blockIdx.x];
  const int first = a.seq_start[s] + row0, n_tok = min(GC_L, a.seq_start[s + 1] - first);
  const int n_qk = a.n_qk(), tid = threadIdx.x, lane = tid & 31;
  const CopyPlan rows_dim(dim);
  gc_load_rows(rows_dim, sK, ld, kn + (size_t)first * n_qk + g * dim, n_qk, n_tok);
  const bool with_qk = !DELTA || h % per_group == 0;
  if (with_qk) gc_load_rows(rows_dim, sQ, ld, qn + (size_t)first * n_qk + g * dim, n_qk, n_tok);
  gc_commit();
  if (DELTA && tid < 32) {
    float l[2], b[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = 2 * lane + e;
      const float* p = lb + ((size_t)(first + t) * a.heads + h) * 2;
      l[e] = t < n_tok ? p[0] : 0.f;
      b[e] = t < n_tok ? p[1] : 0.f;
    }
    const float2 c = gc_cumulate(l[0], l[1], lane);
    sc[2 * lane] = c.x; sc[2 * lane + 1] = c.y;
    sb[2 * lane] = b[0]; sb[2 * lane + 1] = b[1];
  }
  gc_wait();
  __syncthreads();
  const int rg = tid >> 4, cg = tid & 15;  // rows rg + 16 i, columns cg + 16 j
  for (int which = DELTA ? 0 : 1; which < 2; ++which) {  // 0: k . k, 1: q . k
    if (which == 1 && !with_qk) break;
    const float* X = which ? sQ : sK;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int d = 0; d < dim; d += 4) {
      float4 x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) x[i] = *reinterpret_cast<const float4*>(X + (rg + 16 * i) * ld + d);
#pragma unroll
      for (int j = 0; j < 4; ++j) y[j] = *reinterpret_cast<const float4*>(sK + (cg + 16 * j) * ld + d);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (j <= i) {  // column block j beyond row block i lies above the diagonal
            acc[i][j] = fmaf(x[i].x, y[j].x, acc[i][j]); acc[i][j] = fmaf(x[i].y, y[j].y, acc[i][j]);
            acc[i][j] = fmaf(x[i].z, y[j].z, acc[i][j]); acc[i][j] = fmaf(x[i].w, y[j].w, acc[i][j]);
          }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = rg + 16 * i, u = cg + 16 * j;
        if (which == 0) sA[t * GC_PLD + u] = u < t ? sb[t] * expf(sc[t] - sc[u]) * acc[i][j] : 0.f;
        else if (t < n_tok) qk[((size_t)(first + t) * a.groups + g) * GC_L + u] = u <= t ? acc[i][j] : 0.f;
      }
  }
  if (!DELTA) return;
  __syncthreads();
  if (tid < GC_L) {  // a thread per column of the inverse, by forward substitution in registers
    float x[GC_L];
#pragma unroll
    for (int t = 0; t < GC_L; ++t) {
      float p0 = t == tid ? 1.0f : 0.f, p1 = 0.f, p2 = 0.f, p3 = 0.f;
#pragma unroll
      for (int u = 0; u + 3 < t; u += 4) {
        const float4 r = *reinterpret_cast<const float4*>(sA + t * GC_PLD + u);
        p0 = fmaf(-r.x, x[u], p0); p1 = fmaf(-r.y, x[u + 1], p1); p2 = fmaf(-r.z, x[u + 2], p2); p3 = fmaf(-r.w, x[u + 3], p3);
      }
#pragma unroll
      for (int u = t / 4 * 4; u < t; ++u) p0 = fmaf(-sA[t * GC_PLD + u], x[u], p0);
      x[t] = (p0 + p1) + (p2 + p3);
    }
    const float b = sb[tid];
#pragma unroll
    for (int t = 0; t < GC_L; ++t)
      if (t < n_tok) winv[((size_t)(first + t) * a.heads + h) * GC_L + tid] = x[t] * b;
  }
}

template <int N>
__device__ __forceinline__ void gc_read(const float* p, float* o);
template <>
__device__ __forceinline__ void gc_read<4>(const float* p, float* o) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w;
}
template <>
__device__ __forceinline__ void gc_read<2>(const float* p, float* o) {
  const float2 a = *reinterpret_cast<const float2*>(p);
  o[0] = a.x; o[1] = a.y;
}
template <int N>
__device__ __forceinline__ void gc_write(float* p, const float* o);
template <>
__device__ __forceinline__ void gc_write<4>(float* p, const float* o) { *reinterpret_cast<float4*>(p) = make_float4(o[0], o[1], o[2], o[3]); }
template <>
__device__ __forceinline__ void gc_write<2>(float* p, const float* o) { *reinterpret_cast<float2*>(p) = make_float2(o[0], o[1]); }

// acc += row[0 .. end) . U, TC columns; U's rows u_ld apart, end a multiple of four
template <int TC>
__device__ __forceinline__ void gc_row_product(float* acc, const float* row, const float* U, int u_ld, int end) {
  for (int s = 0; s < end; s += 4) {
    const float4 m = *reinterpret_cast<const float4*>(row + s);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float u[TC];
      gc_read<TC>(U + (s + e) * u_ld, u);
      const float f = e == 0 ? m.x : e == 1 ? m.y : e == 2 ? m.z : m.w;
#pragma unroll
      for (int c = 0; c < TC; ++c) acc[c] = fmaf(f, u[c], acc[c]);
    }
  }
}

// Floats of shared memory of the chain's block; the operands that lie token by token (or state row by state row) have rows
// of CT + 8 numbers, which keeps the tensor cores' fragment reads free of bank conflicts.
static size_t gc_smem_floats(bool delta, int dim, int ct, int stages) {
  const int sld = ct + 8;
  return (size_t)stages * 2 * GC_L * (dim + 4) + (size_t)dim * sld + 2 * GC_L * sld + (size_t)stages * GC_L * GC_PLD +
         (delta ? GC_L * GC_PLD : dim * sld) + 4 * GC_L;
}

__device__ __forceinline__ void gc_named_sync(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }
__device__ __forceinline__ void gc_named_arrive(int id, int threads) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

// Single-precision products on the tensor cores: every operand as the sum of two TF32 numbers (its first 11 bits and the
// next 11), three products, float32 sums.  The warp's tile is 16 rows x 8 NT columns; lane = 4 g + q holds the rows g and
// g + 8.
__device__ __forceinline__ void gc_split(float x, unsigned& hi, unsigned& lo) {
  hi = __float_as_uint(x) & 0xffffe000u;
  lo = __float_as_uint(x - __uint_as_float(hi));
}
__device__ __forceinline__ void gc_mma(float* c, const unsigned* a, const unsigned* b) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
// acc += A B over k < k_end (a multiple of eight), pointers at the tile's first row and column: A's element (row, k) at
// A[row * a_ld + k], with A_BY_K at A[k * a_ld + row]; B's (k, column) at B[k * SLD + column].
template <int NT, int SLD, bool A_BY_K>
__device__ __forceinline__ void gc_tile_product(float* acc, const float* A, int a_ld, const float* B, int k_end, int lane) {
  const int g = lane >> 2, q = lane & 3;
  const float* p0 = A + (A_BY_K ? q * a_ld + g : g * a_ld + q);
  const float* p1 = p0 + (A_BY_K ? 4 * a_ld : 8 * a_ld);
  const float* r = B + q * SLD + g;
  const int step = A_BY_K ? 8 * a_ld : 8;
#pragma unroll 2
  for (int k = 0; k < k_end; k += 8) {
    unsigned ah[4], al[4];
    gc_split(p0[0], ah[0], al[0]);
    gc_split(A_BY_K ? p0[8] : p1[0], ah[1], al[1]);
    gc_split(A_BY_K ? p1[0] : p0[4], ah[2], al[2]);
    gc_split(A_BY_K ? p1[8] : p1[4], ah[3], al[3]);
    p0 += step;
    p1 += step;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      unsigned bh[2], bl[2];
      gc_split(r[8 * j], bh[0], bl[0]);
      gc_split(r[8 * j + 4 * SLD], bh[1], bl[1]);
      gc_mma(acc + 4 * j, al, bh);
      gc_mma(acc + 4 * j, ah, bl);
      gc_mma(acc + 4 * j, ah, bh);
    }
    r += 8 * SLD;
  }
}
__device__ __forceinline__ float gc_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Where element e of a thread's CT / 4 results lies in the chunk's [64][CT] matrices (e and e + 1, e even, are neighbours).
template <int CT, bool MMA>
__device__ __forceinline__ int2 gc_place(int t256, int e) {
  if (MMA) {
    const int warp = t256 >> 5, lane = t256 & 31;
    return make_int2((warp >> 1) * 16 + (lane >> 2) + (e & 2 ? 8 : 0), (warp & 1) * (CT / 2) + (e >> 2) * 8 + (lane & 3) * 2 + (e & 1));
  }
  return make_int2((t256 >> 3) + 32 * (e / (CT / 8)), (t256 & 7) * (CT / 8) + e % (CT / 8));
}

// o = X S for the thread's elements: X [64][ld], S [dim][sld]
template <int CT, bool MMA>
__device__ __forceinline__ void gc_state_product(float* o, const float* X, int ld, const float* S, int dim, int t256) {
  constexpr int SLD = CT + 8, TC = CT / 8;
#pragma unroll
  for (int e = 0; e < CT / 4; ++e) o[e] = 0.f;
  if (MMA) {
    const int warp = t256 >> 5;
    gc_tile_product<CT / 16, SLD, false>(o, X + (warp >> 1) * 16 * ld, ld, S + (warp & 1) * (CT / 2), dim, t256 & 31);
    return;
  }
  const int rg = t256 >> 3, cg = t256 & 7;
#pragma unroll 2
  for (int d = 0; d < dim; d += 4) {
    float4 x[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) x[i] = *reinterpret_cast<const float4*>(X + (rg + 32 * i) * ld + d);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float sv[TC];
      gc_read<TC>(S + (d + e) * SLD + cg * TC, sv);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float f = e == 0 ? x[i].x : e == 1 ? x[i].y : e == 2 ? x[i].z : x[i].w;
#pragma unroll
        for (int c = 0; c < TC; ++c) o[i * TC + c] = fmaf(f, sv[c], o[i * TC + c]);
      }
    }
  }
}

// o += M U for the thread's elements: M [64][GC_PLD] lower triangular, U [64][sld]
template <int CT, bool MMA>
__device__ __forceinline__ void gc_chunk_product(float* o, const float* M, const float* U, int t256) {
  constexpr int SLD = CT + 8, TC = CT / 8;
  const int warp = t256 >> 5;
  if (MMA) {
    gc_tile_product<CT / 16, SLD, false>(o, M + (warp >> 1) * 16 * GC_PLD, GC_PLD, U + (warp & 1) * (CT / 2), (warp >> 1) * 16 + 16, t256 & 31);
    return;
  }
  const int rg = t256 >> 3, cg = t256 & 7;
  const int end = warp * 4 + 36;  // the warp's rows are 4 w .. 4 w + 3 and those + 32
  for (int s = 0; s < end; s += 4) {
    float4 m[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) m[i] = *reinterpret_cast<const float4*>(M + (rg + 32 * i) * GC_PLD + s);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float u[TC];
      gc_read<TC>(U + (s + e) * SLD + cg * TC, u);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float f = e == 0 ? m[i].x : e == 1 ? m[i].y : e == 2 ? m[i].z : m[i].w;
#pragma unroll
        for (int c = 0; c < TC; ++c) o[i * TC + c] = fmaf(f, u[c], o[i * TC + c]);
      }
    }
  }
}

// to = carry * from + K^T D by eight warps: K [64][ld], D [64][sld], to and from [dim][sld] (they may be one)
template <int CT, bool MMA>
__device__ __forceinline__ void gc_advance_state(float* to, const float* from, float carry, const float* K, int ld, const float* D, int dim,
                                                 int t256) {
  constexpr int SLD = CT + 8, TC = CT / 8;
  if (MMA) {
    const int lane = t256 & 31, g = lane >> 2, q = lane & 3;
    for (int d0 = (t256 >> 5) * 16; d0 < dim; d0 += 128) {
      float acc[CT / 2];
#pragma unroll
      for (int e = 0; e < CT / 2; ++e) acc[e] = 0.f;
      gc_tile_product<CT / 8, SLD, true>(acc, K + d0, ld, D, GC_L, lane);
#pragma unroll
      for (int e = 0; e < CT / 2; e += 2) {
        const int d = d0 + g + (e & 2 ? 8 : 0), at = d * SLD + (e >> 2) * 8 + 2 * q;
        if (d < dim) {
          float old[2];
          gc_read<2>(from + at, old);
          old[0] = fmaf(carry, old[0], acc[e]);
          old[1] = fmaf(carry, old[1], acc[e + 1]);
          gc_write<2>(to + at, old);
        }
      }
    }
    return;
  }
  const int rg = t256 >> 3, cg = t256 & 7;
  for (int d = rg * 4; d < dim; d += 128) {
    float acc[4][TC];
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
      for (int c = 0; c < TC; ++c) acc[e][c] = 0.f;
#pragma unroll 4
    for (int t = 0; t < GC_L; ++t) {
      const float4 k = *reinterpret_cast<const float4*>(K + t * ld + d);
      float u[TC];
      gc_read<TC>(D + t * SLD + cg * TC, u);
#pragma unroll
      for (int c = 0; c < TC; ++c) {
        acc[0][c] = fmaf(k.x, u[c], acc[0][c]);
        acc[1][c] = fmaf(k.y, u[c], acc[1][c]);
        acc[2][c] = fmaf(k.z, u[c], acc[2][c]);
        acc[3][c] = fmaf(k.w, u[c], acc[3][c]);
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float old[TC];
      gc_read<TC>(from + (d + e) * SLD + cg * TC, old);
#pragma unroll
      for (int c = 0; c < TC; ++c) old[c] = fmaf(carry, old[c], acc[e][c]);
      gc_write<TC>(to + (d + e) * SLD + cg * TC, old);
    }
  }
}

// The chain: one block per (sequence, head, CT value columns), two halves of eight warps.  A thread of either half has CT / 4
// elements of the chunk's [64][CT] matrices (gc_place).  The second half makes the outputs, Q S0 and P U; the first
// advances the state, in the delta rule after it has made the right-hand sides V - e^c K S0 and both halves have
// multiplied them into U.  Without a delta rule the halves meet once per chunk: the state goes into a buffer of its own while
// the other half still reads the old one.  With two stages the next chunk's rows arrive while this one's are worked on.
// MMA: the products on the tensor cores (dim a multiple of eight), else on the CUDA cores.
template <typename T, bool DELTA, int CT, bool MMA>
__global__ void __launch_bounds__(GC_CHAIN_THREADS) gated_state_chunk_kernel(const GatedStateArgs a, const float* __restrict__ qn,
                                                                             const float* __restrict__ kn, const float* __restrict__ vc,
                                                                             const float* __restrict__ lb, const float* __restrict__ qk,
                                                                             const float* __restrict__ winv, int col_tiles, int stages,
                                                                             float* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int TC = CT / 8, NE = CT / 4, SLD = CT + 8;
  extern __shared__ __align__(16) float sm[];
  const int heads = a.heads, dim = a.dim, vdim = a.vdim, ld = dim + 4, n_qk = a.n_qk();
  float* sKQ = sm;                                        // [stages][K 64 rows | Q 64 rows][ld]
  float* sS = sKQ + (size_t)stages * 2 * GC_L * ld;       // [dim][SLD]
  float* sU = sS + (size_t)dim * SLD;                     // [64][SLD] u
  float* sD = sU + GC_L * SLD;                            // [64][SLD] right-hand sides; u times its weight in the state after the chunk
  float* sP = sD + GC_L * SLD;                            // [stages][64][GC_PLD]
  float* sW = sP + (size_t)stages * GC_L * GC_PLD;        // delta: [64][GC_PLD]
  float* sS2 = sW;                                        // otherwise: [dim][SLD], the state after the chunk
  float* sc = sW + (DELTA ? GC_L * GC_PLD : dim * SLD);   // [64] c, then b, e^c, e^(c_end - c)
  float *sb = sc + GC_L, *se = sb + GC_L, *sd = se + GC_L;
  const int tile = blockIdx.x % col_tiles, h = (blockIdx.x / col_tiles) % heads, s = blockIdx.x / (col_tiles * heads);
  const int per_group = heads / a.groups, g = h / per_group;
  const int tid = threadIdx.x, t256 = tid & 255, lane = tid & 31;
  const bool outputs = tid >= 256;  // the second half
  const int col0 = tile * CT;
  const int start = a.seq_start[s], n = a.seq_start[s + 1] - start;
  float* S_g = a.state + (size_t)a.slots[s] * a.state_stride + (size_t)h * dim * vdim;
  for (int i = tid; i < dim * CT; i += GC_CHAIN_THREADS) {
    const int d = i / CT, c = i - d * CT;
    sS[d * SLD + c] = col0 + c < vdim ? S_g[(size_t)d * vdim + col0 + c] : 0.f;
  }
  const float skip = a.d ? a.d[h] : 0.f;
  const CopyPlan rows_dim(dim), rows_64(GC_L);
  auto load_kq = [&](int base, int stage) {
    float* dst = sKQ + (size_t)stage * 2 * GC_L * ld;
    const int left = min(GC_L, n - base);
    gc_load_rows(rows_dim, dst, ld, kn + (size_t)(start + base) * n_qk + g * dim, n_qk, left);
    gc_load_rows(rows_dim, dst + GC_L * ld, ld, qn + (size_t)(start + base) * n_qk + g * dim, n_qk, left);
    gc_load_rows(rows_64, sP + (size_t)stage * GC_L * GC_PLD, GC_PLD, qk + ((size_t)(start + base) * a.groups + g) * GC_L,
                 (size_t)a.groups * GC_L, left);
  };
  auto load_w = [&](int base) {
    gc_load_rows(rows_64, sW, GC_PLD, winv + ((size_t)(start + base) * heads + h) * GC_L, (size_t)heads * GC_L, min(GC_L, n - base));
  };
  const bool pairs = vdim % 2 == 0 && (((uintptr_t)vc | (uintptr_t)out) & 7) == 0;
  float v_next[NE], l_next[2] = {0.f, 0.f}, b_next[2] = {0.f, 0.f};
  auto load_v = [&](int base) {
#pragma unroll
    for (int e = 0; e < NE; e += 2) {
      const int2 at = gc_place<CT, MMA>(t256, e);
      const int t = base + at.x, col = col0 + at.y;
      const float* p = vc + (size_t)(start + t) * heads * vdim + (size_t)h * vdim + col;
      if (pairs && t < n && col < vdim) {
        gc_read<2>(p, v_next + e);
      } else {
        v_next[e] = t < n && col < vdim ? p[0] : 0.f;
        v_next[e + 1] = t < n && col + 1 < vdim ? p[1] : 0.f;
      }
    }
    if (tid < 32) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = base + 2 * lane + e;
        const float* p = lb + ((size_t)(start + t) * heads + h) * 2;
        l_next[e] = t < n ? p[0] : 0.f;
        b_next[e] = t < n ? p[1] : 0.f;
      }
    }
  };
  if (stages == 2) load_kq(0, 0);
  if (DELTA) load_w(0);
  gc_commit();
  load_v(0);
  for (int base = 0, stage = 0; base < n; base += GC_L, stage ^= stages - 1) {
    __syncthreads();  // the chunk before is done with everything in shared memory
    if (stages == 1) {
      load_kq(base, 0);
      gc_commit();
    }
    if (tid < 32) {
      const float2 c = gc_cumulate(l_next[0], l_next[1], lane);
      const float end = __shfl_sync(0xffffffffu, c.y, 31);  // tokens past the end have log decay 0
      sc[2 * lane] = c.x; sc[2 * lane + 1] = c.y;
      sb[2 * lane] = b_next[0]; sb[2 * lane + 1] = b_next[1];
      se[2 * lane] = expf(c.x); se[2 * lane + 1] = expf(c.y);
      sd[2 * lane] = expf(end - c.x); sd[2 * lane + 1] = expf(end - c.y);
    }
    float v[NE];
#pragma unroll
    for (int e = 0; e < NE; ++e) v[e] = v_next[e];
    gc_wait();
    __syncthreads();
    const bool more = base + GC_L < n;
    if (more) {
      if (stages == 2) {
        load_kq(base + GC_L, stage ^ 1);
        gc_commit();
      }
      load_v(base + GC_L);
    }
    const float* K = sKQ + (size_t)stage * 2 * GC_L * ld;
    float* P = sP + (size_t)stage * GC_L * GC_PLD;
    float o[NE];
    if (outputs) {
      // the decays onto q . k (above the diagonal the first kernel left zeros), then Q S0
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = (t256 >> 4) + 16 * j, u = (t256 & 15) * 4;
        if (u <= t) {
          float p[4], c[4];
          gc_read<4>(P + t * GC_PLD + u, p);
          gc_read<4>(sc + u, c);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float x = fminf(sc[t] - c[e], 0.f);  // above the diagonal p is zero
            p[e] *= MMA ? gc_ex2(x * 1.4426950408889634f) : expf(x);
          }
          gc_write<4>(P + t * GC_PLD + u, p);
        }
      }
      gc_state_product<CT, MMA>(o, K + GC_L * ld, ld, sS, dim, t256);
#pragma unroll
      for (int e = 0; e < NE; ++e) o[e] *= se[gc_place<CT, MMA>(t256, e).x];
    } else if (DELTA) {
      gc_state_product<CT, MMA>(o, K, ld, sS, dim, t256);
#pragma unroll
      for (int e = 0; e < NE; e += 2) {
        const int2 at = gc_place<CT, MMA>(t256, e);
        const float r[2] = {v[e] - o[e] * se[at.x], v[e + 1] - o[e + 1] * se[at.x]};
        gc_write<2>(sD + at.x * SLD + at.y, r);
      }
    } else {
#pragma unroll
      for (int e = 0; e < NE; e += 2) {
        const int2 at = gc_place<CT, MMA>(t256, e);
        const float u[2] = {v[e] * sb[at.x], v[e + 1] * sb[at.x]}, w[2] = {u[0] * sd[at.x], u[1] * sd[at.x]};
        gc_write<2>(sU + at.x * SLD + at.y, u);
        gc_write<2>(sD + at.x * SLD + at.y, w);
      }
      gc_named_arrive(2, GC_CHAIN_THREADS);  // the other half may read u
      gc_named_sync(1, 256);
      gc_advance_state<CT, MMA>(sS2, sS, se[GC_L - 1], K, ld, sD, dim, t256);
    }
    if (DELTA) {
      __syncthreads();
      // U = W R over both halves: a tile of 16 x 8 per warp, or a token and TC columns per thread
      constexpr int UE = MMA ? 4 : TC;
      const int warp = tid >> 5;
      const bool has_u = !MMA || (warp & 3) * 8 < CT;
      float u[UE];
#pragma unroll
      for (int e = 0; e < UE; ++e) u[e] = 0.f;
      if (MMA) {
        if (has_u)
          gc_tile_product<1, SLD, false>(u, sW + (warp >> 2) * 16 * GC_PLD, GC_PLD, sD + (warp & 3) * 8, (warp >> 2) * 16 + 16, lane);
      } else {
        gc_row_product<TC>(u, sW + (tid >> 3) * GC_PLD, sD + (tid & 7) * TC, SLD, (warp + 1) * 4);
      }
      __syncthreads();  // the right-hand sides have been read
      if (has_u) {
#pragma unroll
        for (int e = 0; e < UE; e += 2) {
          const int t = MMA ? (warp >> 2) * 16 + (lane >> 2) + (e & 2 ? 8 : 0) : tid >> 3;
          const int at = t * SLD + (MMA ? (warp & 3) * 8 + (lane & 3) * 2 : (tid & 7) * TC + e);
          const float w[2] = {u[e] * sd[t], u[e + 1] * sd[t]};
          gc_write<2>(sU + at, u + e);
          gc_write<2>(sD + at, w);
        }
      }
      __syncthreads();
      if (more) {
        load_w(base + GC_L);
        gc_commit();
      }
      if (!outputs) gc_advance_state<CT, MMA>(sS, sS, se[GC_L - 1], K, ld, sD, dim, t256);
    } else if (outputs) {
      gc_named_sync(2, GC_CHAIN_THREADS);  // u, and this half's decays
    }
    if (outputs) {
      gc_chunk_product<CT, MMA>(o, P, sU, t256);
#pragma unroll
      for (int e = 0; e < NE; e += 2) {
        const int2 at = gc_place<CT, MMA>(t256, e);
        const int t = base + at.x, col = col0 + at.y;
        if (t < n && col < vdim) {
          float* dst = out + (size_t)(start + t) * heads * vdim + (size_t)h * vdim + col;
          const float y[2] = {fmaf(skip, v[e], o[e]), fmaf(skip, v[e + 1], o[e + 1])};
          if (pairs) {
            gc_write<2>(dst, y);
          } else {
            dst[0] = y[0];
            if (col + 1 < vdim) dst[1] = y[1];
          }
        }
      }
    }
    if (!DELTA) {
      float* swap = sS;
      sS = sS2;
      sS2 = swap;
    }
  }
  __syncthreads();
  for (int i = tid; i < dim * CT; i += GC_CHAIN_THREADS) {
    const int d = i / CT, c = i - d * CT;
    if (col0 + c < vdim) S_g[(size_t)d * vdim + col0 + c] = sS[d * SLD + c];
  }
  gs_keep_inputs<T>(a, s, h, col0, min(CT, vdim - col0), tile == 0 && h % per_group == 0);
}

// Steps of one token per sequence: convolution, gates, unit norms, one step of the recurrence and the ring in one
// launch.  Blocks as above; each of them convolves its group's q and k channels itself.
template <typename T, int RW, bool DELTA>
__global__ void __launch_bounds__(GS_THREADS) gated_state_token_kernel(const GatedStateArgs a, int col_tiles, float* __restrict__ out) {
  pdl_launch_dependents();
  constexpr int ROWS = GS_WARPS * RW;
  __shared__ __align__(16) float in[2 * ROWS + 32];  // q, k, the block's values
  __shared__ float red[GS_WARPS][65];
  __shared__ float norms[2];
  const int heads = a.heads, dim = a.dim, vdim = a.vdim;
  const int tile = blockIdx.x % col_tiles, h = (blockIdx.x / col_tiles) % heads, s = blockIdx.x / (col_tiles * heads);
  const int per_group = heads / a.groups, g = h / per_group;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int col = tile * 32 + lane, cols = min(32, vdim - tile * 32);
  const bool live = col < vdim;
  const int row0 = warp * RW, n_qk = a.n_qk(), n_ch = a.n_ch();
  pdl_wait();
  const int t = a.seq_start[s], pos = a.seq_pos0[s];
  float* S_g = a.state + (size_t)a.slots[s] * a.state_stride + (size_t)h * dim * vdim;
  float S[RW];
#pragma unroll
  for (int i = 0; i < RW; ++i) S[i] = (live && row0 + i < dim) ? S_g[(size_t)(row0 + i) * vdim + col] : 0.f;
  const float2 gate = gs_gates<DELTA>(a, t, h);
  const T* row = (const T*)a.proj + (size_t)t * a.stride;
  float* ring = const_cast<float*>(a.ring(s));
  const bool keep_qk = tile == 0 && h % per_group == 0;
  for (int i = threadIdx.x; i < 2 * ROWS + 32; i += GS_THREADS) {
    const int which = i / ROWS, d = i - which * ROWS;  // 0: q, 1: k, 2: values
    float y = 0.f;
    if (which < 2 ? d < dim : d < cols) {
      const int c = which == 0 ? g * dim + d : (which == 1 ? n_qk + g * dim + d : 2 * n_qk + h * vdim + tile * 32 + d);
      const float x = to_f32<T>(row[a.column(c)]);
      float acc = fmaf(a.conv_w ? a.conv_w[(size_t)(a.taps - 1) * n_ch + c] : 1.0f, x, a.conv_b ? a.conv_b[c] : 0.f);
      for (int j = 0; j < a.taps - 1; ++j) {
        const int p = pos - (a.taps - 1 - j);
        if (p >= 0) acc = fmaf(a.conv_w[(size_t)j * n_ch + c], ring[(size_t)(p % a.taps) * n_ch + c], acc);
      }
      if (a.taps > 1 && (which == 2 || keep_qk)) ring[(size_t)(pos % a.taps) * n_ch + c] = x;
      y = gs_silu(acc);
    }
    in[i] = y;
  }
  __syncthreads();
  if (DELTA) {
    if (warp < 2) {
      float ss = 0.f;
      for (int i = lane; i < ROWS; i += 32) ss = fmaf(in[warp * ROWS + i], in[warp * ROWS + i], ss);
      ss = warp_sum(ss);
      if (lane == 0) norms[warp] = (1.0f / sqrtf(ss + 1e-6f)) * (warp == 0 ? a.q_scale : 1.0f);
    }
    __syncthreads();
  }
  const float qs = DELTA ? norms[0] : 1.0f, ks = DELTA ? norms[1] : 1.0f;
  const float decay = expf(gate.x), v = in[2 * ROWS + lane];
  float pk = 0.f, pq = 0.f, kq = 0.f;
  float kreg[RW];
#pragma unroll
  for (int i = 0; i < RW; ++i) {
    const float q = in[row0 + i] * qs, k = in[ROWS + row0 + i] * ks;
    S[i] *= decay;
    kreg[i] = k;
    if (DELTA) pk = fmaf(S[i], k, pk);
    pq = fmaf(S[i], q, pq);
    kq = fmaf(k, q, kq);
  }
  if (DELTA) red[warp][lane] = pk;
  red[warp][32 + lane] = pq;
  if (lane == 0) red[warp][64] = kq;
  __syncthreads();
  float sk = 0.f, sq = 0.f, skq = 0.f;
#pragma unroll
  for (int w = 0; w < GS_WARPS; ++w) {
    if (DELTA) sk += red[w][lane];
    sq += red[w][32 + lane];
    skq += red[w][64];
  }
  const float u = gate.y * (v - sk);
  if (live) {
#pragma unroll
    for (int i = 0; i < RW; ++i)
      if (row0 + i < dim) S_g[(size_t)(row0 + i) * vdim + col] = fmaf(kreg[i], u, S[i]);
    if (warp == 0) out[(size_t)t * heads * vdim + (size_t)h * vdim + col] = fmaf(a.d ? a.d[h] : 0.f, v, fmaf(skq, u, sq));
  }
}

static bool gs_fits(const GatedStateArgs& a) {
  const int n_qk = a.groups * a.dim, n_v = a.heads * a.vdim;
  const bool gates = a.log_decay || (a.gate && a.dt_bias && a.a_log && a.a_off >= 0 && a.a_off + a.heads <= a.gate_stride &&
                                     a.b_off + a.heads <= a.gate_stride);
  return a.proj && gates && (a.conv_w || a.taps == 1) && a.state && a.tok_seq && a.seq_start && a.seq_pos0 && a.slots &&
         a.groups > 0 && a.heads > 0 && a.heads % a.groups == 0 && a.dim > 0 && a.dim <= 256 && a.vdim > 0 && a.taps >= 1 &&
         a.taps <= GS_MAX_TAPS && a.q_off >= 0 && a.k_off >= 0 && a.v_off >= 0 && a.q_off + n_qk <= a.stride &&
         a.k_off + n_qk <= a.stride && a.v_off + n_v <= a.stride &&
         a.state_stride >= (size_t)a.heads * a.dim * a.vdim + (a.taps > 1 ? (size_t)a.taps * (2 * n_qk + n_v) : 0);
}

static GatedStateArgs gs_args(const void* proj, int n_tokens, int stride, int q_off, int k_off, int v_off, const float* gate,
                              int gate_stride, int a_off, int b_off, int groups, int heads, int dim, int vdim, int taps,
                              const float* conv_w, const float* conv_b, const float* dt_bias, const float* a_log, const float* d,
                              const float* log_decay, float q_scale, float* state, long long state_stride, const int* tok_seq, const int* seq_start,
                              const int* seq_pos0, const int* slots, int n_seqs) {
  GatedStateArgs a = {};
  a.proj = proj; a.gate = gate; a.conv_w = conv_w; a.conv_b = conv_b; a.dt_bias = dt_bias; a.a_log = a_log; a.d = d; a.log_decay = log_decay;
  a.state = state; a.tok_seq = tok_seq; a.seq_start = seq_start; a.seq_pos0 = seq_pos0; a.slots = slots;
  a.state_stride = (size_t)state_stride; a.q_scale = q_scale; a.stride = stride; a.gate_stride = gate_stride; a.q_off = q_off;
  a.k_off = k_off; a.v_off = v_off; a.a_off = a_off; a.b_off = b_off < 0 ? 0 : b_off; a.groups = groups; a.heads = heads; a.dim = dim;
  a.vdim = vdim; a.taps = taps; a.n_seqs = n_seqs; a.n_tokens = n_tokens;
  return a;
}

// The arguments all entry points share (b_off < 0: the state-space update, or with log_decay the one under fixed decays; else
// the delta rule).
#define GS_PARAMS                                                                                                              \
  const void *proj, int dtype, int n_tokens, int stride, int q_off, int k_off, int v_off, const float *gate, int gate_stride,  \
      int a_off, int b_off, int groups, int heads, int dim, int vdim, int taps, const float *conv_w, const float *conv_b,      \
      const float *dt_bias, const float *a_log, const float *d, const float *log_decay, float q_scale, float *state, long long state_stride,           \
      const int *tok_seq, const int *seq_start, const int *seq_pos0, const int *slots, int n_seqs
#define GS_PASS                                                                                                                \
  proj, n_tokens, stride, q_off, k_off, v_off, gate, gate_stride, a_off, b_off, groups, heads, dim, vdim, taps, conv_w, conv_b, \
      dt_bias, a_log, d, log_decay, q_scale, state, state_stride, tok_seq, seq_start, seq_pos0, slots, n_seqs

// q and k as they enter the recurrence, v, and (log decay, factor) per head, all float32.
extern "C" int bn_gated_state_prepare(GS_PARAMS, float* qn, float* kn, float* vc, float* lb, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  const GatedStateArgs a = gs_args(GS_PASS);
  const bool delta = b_off >= 0;
  const size_t smem = delta ? (size_t)2 * groups * dim * sizeof(float) : 0;
  if (!gs_fits(a) || !qn || !kn || !vc || !lb || smem > 200 * 1024) return BN_ERR_BAD_ARG;
  const bool vec = dim % 4 == 0 && (heads * vdim) % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 &&
                   stride % 4 == 0 && state_stride % 4 == 0 &&
                   !(((uintptr_t)proj | (uintptr_t)conv_w | (uintptr_t)conv_b | (uintptr_t)state | (uintptr_t)qn | (uintptr_t)kn |
                      (uintptr_t)vc) & 15);
#define GS_PREP(TT, VV, DD)                                                                                                        \
  do {                                                                                                                             \
    if (smem > 48 * 1024) {                                                                                                        \
      static size_t granted = 0;                                                                                                   \
      if (smem > granted) {                                                                                                        \
        cudaError_t e = cudaFuncSetAttribute(gated_state_prepare_kernel<TT, VV, DD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e != cudaSuccess) return BN_ERR_LAUNCH + (int)e;                                                                       \
        granted = smem;                                                                                                            \
      }                                                                                                                            \
    }                                                                                                                              \
    BN_LAUNCH((gated_state_prepare_kernel<TT, VV, DD>), n_tokens, 256, smem, stream, a, qn, kn, vc, lb);                           \
  } while (0)
#define GS_PREP_T(TT)                                             \
  do {                                                            \
    if (delta) { if (vec) GS_PREP(TT, 4, true); else GS_PREP(TT, 1, true); } \
    else { if (vec) GS_PREP(TT, 4, false); else GS_PREP(TT, 1, false); }     \
  } while (0)
  if (dtype == BN_F32) GS_PREP_T(float);
  else if (dtype == BN_BF16) GS_PREP_T(__nv_bfloat16);
  else return BN_ERR_BAD_ARG;
#undef GS_PREP_T
#undef GS_PREP
  return BN_OK;
}

#define GS_BY_SIZE(RUN, TT)                                       \
  do {                                                            \
    if (delta) {                                                  \
      if (dim <= 32) RUN(TT, 4, true);                            \
      else if (dim <= 64) RUN(TT, 8, true);                       \
      else if (dim <= 128) RUN(TT, 16, true);                     \
      else RUN(TT, 32, true);                                     \
    } else {                                                      \
      if (dim <= 32) RUN(TT, 4, false);                           \
      else if (dim <= 64) RUN(TT, 8, false);                      \
      else if (dim <= 128) RUN(TT, 16, false);                    \
      else RUN(TT, 32, false);                                    \
    }                                                             \
  } while (0)

// The recurrence over runs of tokens, behind bn_gated_state_prepare; out [T, heads * vdim] float32.
extern "C" int bn_gated_state_run(GS_PARAMS, const float* qn, const float* kn, const float* vc, const float* lb, float* out,
                                  cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return BN_OK;
  const GatedStateArgs a = gs_args(GS_PASS);
  if (!gs_fits(a) || !qn || !kn || !vc || !lb || !out) return BN_ERR_BAD_ARG;
  const bool delta = b_off >= 0;
  const int col_tiles = (vdim + 31) / 32;
  const long long blocks = (long long)n_seqs * heads * col_tiles;
  if (blocks > 2147483647LL) return BN_ERR_BAD_ARG;
#define GS_RUN(TT, RW, DD) \
  BN_LAUNCH((gated_state_kernel<TT, RW, DD>), (unsigned)blocks, GS_THREADS, 0, stream, a, qn, kn, vc, lb, col_tiles, out)
  if (dtype == BN_F32) GS_BY_SIZE(GS_RUN, float);
  else if (dtype == BN_BF16) GS_BY_SIZE(GS_RUN, __nv_bfloat16);
  else return BN_ERR_BAD_ARG;
#undef GS_RUN
  return BN_OK;
}

// As bn_gated_state_run, by chunks of 64 tokens (for steps that bring runs of many tokens; dim a multiple of four).
// tile_seq / tile_row0: the sequence and first row of every run of 64 new tokens.  qk [T, groups, 64] and, for the delta
// rule, winv [T, heads, 64] are working space.
extern "C" int bn_gated_state_chunks(GS_PARAMS, const float* qn, const float* kn, const float* vc, const float* lb, const int* tile_seq,
                                     const int* tile_row0, int n_tiles, float* qk, float* winv, float* out, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return BN_OK;
  const GatedStateArgs a = gs_args(GS_PASS);
  const bool delta = b_off >= 0;
  if (!gs_fits(a) || !qn || !kn || !vc || !lb || !out || !tile_seq || !tile_row0 || n_tiles <= 0 || !qk || (delta && !winv) || dim % 4 ||
      heads > 65535 || (((uintptr_t)qn | (uintptr_t)kn | (uintptr_t)qk | (uintptr_t)winv) & 15))
    return BN_ERR_BAD_ARG;
  const size_t local = ((size_t)(2 * GC_L) * (dim + 4) + (delta ? GC_L * GC_PLD : 0)) * sizeof(float);
  if (local > 200 * 1024) return BN_ERR_BAD_ARG;
  static size_t granted_local[2] = {0, 0};
  if (local > 48 * 1024 && local > granted_local[delta]) {
    cudaError_t e = delta ? cudaFuncSetAttribute(gated_state_local_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)local)
                          : cudaFuncSetAttribute(gated_state_local_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)local);
    if (e != cudaSuccess) return BN_ERR_LAUNCH + (int)e;
    granted_local[delta] = local;
  }
  if (delta)
    BN_LAUNCH(gated_state_local_kernel<true>, dim3(n_tiles, heads), GC_THREADS, local, stream, a, qn, kn, lb, tile_seq, tile_row0, qk, winv);
  else
    BN_LAUNCH(gated_state_local_kernel<false>, dim3(n_tiles, groups), GC_THREADS, local, stream, a, qn, kn, lb, tile_seq, tile_row0, qk, winv);
  // 32 columns per block, or 16 where that leaves most of the SMs without one (or a block's memory too small)
  const size_t most = 227 * 1024;  // shared memory of a block
  const bool fits32 = gc_smem_floats(delta, dim, 32, 1) * sizeof(float) <= most;
  const int ct = fits32 && (long long)n_seqs * heads * ((vdim + 31) / 32) >= 100 ? 32 : 16;
  const int col_tiles = (vdim + ct - 1) / ct;
  const int stages = gc_smem_floats(delta, dim, ct, 2) * sizeof(float) <= most ? 2 : 1;
  const size_t smem = gc_smem_floats(delta, dim, ct, stages) * sizeof(float);
  const long long blocks = (long long)n_seqs * heads * col_tiles;
  if (smem > most || blocks > 2147483647LL) return BN_ERR_BAD_ARG;
#define GC_RUN(TT, DD, CC, MM)                                                                                                           \
  do {                                                                                                                                   \
    static size_t granted = 0;                                                                                                           \
    if (smem > granted) {                                                                                                                \
      cudaError_t e = cudaFuncSetAttribute(gated_state_chunk_kernel<TT, DD, CC, MM>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (e != cudaSuccess) return BN_ERR_LAUNCH + (int)e;                                                                               \
      granted = smem;                                                                                                                    \
    }                                                                                                                                    \
    BN_LAUNCH((gated_state_chunk_kernel<TT, DD, CC, MM>), (unsigned)blocks, GC_CHAIN_THREADS, smem, stream, a, qn, kn, vc, lb, qk, winv, \
              col_tiles, stages, out);                                                                                                   \
  } while (0)
#define GC_RUN_T(TT, MM)                                                                           \
  do {                                                                                             \
    if (delta) { if (ct == 32) GC_RUN(TT, true, 32, MM); else GC_RUN(TT, true, 16, MM); }          \
    else { if (ct == 32) GC_RUN(TT, false, 32, MM); else GC_RUN(TT, false, 16, MM); }              \
  } while (0)
  // the float32 path keeps to the CUDA cores
  if (dtype == BN_F32) GC_RUN_T(float, false);
  else if (dtype == BN_BF16 && dim % 8 == 0) GC_RUN_T(__nv_bfloat16, true);
  else if (dtype == BN_BF16) GC_RUN_T(__nv_bfloat16, false);
  else return BN_ERR_BAD_ARG;
#undef GC_RUN_T
#undef GC_RUN
  return BN_OK;
}

// One token per sequence, from the projection to the recurrence's output in one launch.
extern "C" int bn_gated_state_token(GS_PARAMS, float* out, cudaStream_t stream) {
  if (n_tokens <= 0 || n_seqs <= 0) return BN_OK;
  const GatedStateArgs a = gs_args(GS_PASS);
  if (!gs_fits(a) || !out || n_tokens != n_seqs) return BN_ERR_BAD_ARG;
  const bool delta = b_off >= 0;
  const int col_tiles = (vdim + 31) / 32;
  const long long blocks = (long long)n_seqs * heads * col_tiles;
  if (blocks > 2147483647LL) return BN_ERR_BAD_ARG;
#define GS_TOKEN(TT, RW, DD) \
  BN_LAUNCH((gated_state_token_kernel<TT, RW, DD>), (unsigned)blocks, GS_THREADS, 0, stream, a, col_tiles, out)
  if (dtype == BN_F32) GS_BY_SIZE(GS_TOKEN, float);
  else if (dtype == BN_BF16) GS_BY_SIZE(GS_TOKEN, __nv_bfloat16);
  else return BN_ERR_BAD_ARG;
#undef GS_TOKEN
  return BN_OK;
}

// ---- behind the recurrence --------------------------------------------------------------------------
// Every row of o [T, parts * len] in equal parts, with a gate z of the same width:
//   gate first   y = o silu(z);            out = y / sqrt(mean over the part (y^2) + eps) * gain
//   gate last    out = o / sqrt(mean over the part (o^2) + eps) * gain * silu(z), or * sigmoid(z)
// gain holds one number per place of the row, or per place of a part (gain_len = len: shared by the parts).
// THREADS 32: a warp per part, eight parts per block; else a block per part.  The part waits in shared memory.
template <typename T, typename G, int THREADS, int V>
__global__ void state_output_kernel(const float* __restrict__ o, const G* __restrict__ z, int z_stride, const float* __restrict__ gain,
                                    int gain_len, int parts, int len, float eps, int gate_first, int logistic, T* __restrict__ out, int n_items) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float part[];
  __shared__ float scratch[32];
  const int sub = THREADS == 32 ? threadIdx.x >> 5 : 0, lane = THREADS == 32 ? threadIdx.x & 31 : threadIdx.x;
  const int step = (THREADS == 32 ? 32 : blockDim.x) * V;
  const int item = THREADS == 32 ? blockIdx.x * (blockDim.x >> 5) + sub : blockIdx.x;
  if (item >= n_items) return;
  const int t = item / parts, p = item - t * parts;
  float* y = part + (size_t)sub * ((len + 3) / 4 * 4);
  const float* os = o + (size_t)item * len;
  const G* zs = z + (size_t)t * z_stride + (size_t)p * len;
  float ss = 0.f;
  for (int i = lane * V; i < len; i += step) {
    float a[V], g[V];
    gs_load<float, V>(os + i, a);
    if (gate_first) {
      gs_load<G, V>(zs + i, g);
#pragma unroll
      for (int e = 0; e < V; ++e) a[e] *= gs_silu(g[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      y[i + e] = a[e];
      ss = fmaf(a[e], a[e], ss);
    }
  }
  ss = THREADS == 32 ? warp_sum(ss) : block_sum(ss, scratch);
  const float scale = 1.0f / sqrtf(ss / (float)len + eps);
  const float* gn = gain + (gain_len == len ? 0 : (size_t)p * len);
  T* dst = out + (size_t)item * len;
  for (int i = lane * V; i < len; i += step) {
    float g[V], w[V];
    gs_load<float, V>(gn + i, w);
    if (!gate_first) gs_load<G, V>(zs + i, g);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      w[e] *= y[i + e] * scale;
      if (!gate_first) w[e] *= logistic ? 1.0f / (1.0f + expf(-g[e])) : gs_silu(g[e]);
    }
    if (V == 4 && sizeof(T) == 2) {
      const __nv_bfloat162 a = __floats2bfloat162_rn(w[0], w[1 % V]), b = __floats2bfloat162_rn(w[2 % V], w[3 % V]);
      uint2 raw;
      raw.x = *reinterpret_cast<const unsigned*>(&a);
      raw.y = *reinterpret_cast<const unsigned*>(&b);
      *reinterpret_cast<uint2*>(dst + i) = raw;
    } else if (V == 4) {
      *reinterpret_cast<float4*>(dst + i) = make_float4(w[0], w[1 % V], w[2 % V], w[3 % V]);
    } else {
      dst[i] = from_f32<T>(w[0]);
    }
  }
}

template <typename T, typename G, int THREADS, int V>
static int launch_state_output(const float* o, const void* z, int z_stride, const float* gain, int gain_len, int parts, int len,
                               float eps, int gate_first, int logistic, void* out, int n_items, cudaStream_t stream) {
  const int padded = (len + 3) / 4 * 4;
  const size_t smem = (size_t)padded * sizeof(float) * (THREADS == 32 ? 8 : 1);
  if (smem > 200 * 1024) return BN_ERR_BAD_ARG;
  if (smem > 48 * 1024) {
    static size_t granted = 0;
    if (smem > granted) {
      cudaError_t e = cudaFuncSetAttribute(state_output_kernel<T, G, THREADS, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return BN_ERR_LAUNCH + (int)e;
      granted = smem;
    }
  }
  const unsigned blocks = THREADS == 32 ? (unsigned)((n_items + 7) / 8) : (unsigned)n_items;
  const int threads = THREADS == 32 ? 256 : (len >= 4096 ? 512 : 256);
  BN_LAUNCH((state_output_kernel<T, G, THREADS, V>), blocks, threads, smem, stream, o, (const G*)z, z_stride, gain, gain_len, parts, len,
            eps, gate_first, logistic, (T*)out, n_items);
  return BN_OK;
}

extern "C" int bn_state_output(const float* o, const void* z, int z_dtype, int z_stride, const float* gain, int gain_len, int dtype,
                               int n_tokens, int parts, int len, float eps, int gate_first, int logistic, void* out, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  if (!o || !z || !gain || !out || parts <= 0 || len <= 0 || z_stride < parts * len || !(eps > 0.f) || (gate_first && logistic) ||
      (gain_len != len && gain_len != parts * len))
    return BN_ERR_BAD_ARG;
  const int items = n_tokens * parts;
  const bool vec = len % 4 == 0 && z_stride % 4 == 0 && !(((uintptr_t)o | (uintptr_t)z | (uintptr_t)gain | (uintptr_t)out) & 15);
#define GS_OUT(TT, GG)                                                                                                               \
  do {                                                                                                                               \
    if (len <= 512)                                                                                                                  \
      return vec ? launch_state_output<TT, GG, 32, 4>(o, z, z_stride, gain, gain_len, parts, len, eps, gate_first, logistic, out, items, stream) \
                 : launch_state_output<TT, GG, 32, 1>(o, z, z_stride, gain, gain_len, parts, len, eps, gate_first, logistic, out, items, stream); \
    return vec ? launch_state_output<TT, GG, 256, 4>(o, z, z_stride, gain, gain_len, parts, len, eps, gate_first, logistic, out, items, stream) \
               : launch_state_output<TT, GG, 256, 1>(o, z, z_stride, gain, gain_len, parts, len, eps, gate_first, logistic, out, items, stream); \
  } while (0)
  if (dtype == BN_F32 && z_dtype == BN_F32) GS_OUT(float, float);
  if (dtype == BN_BF16 && z_dtype == BN_F32) GS_OUT(__nv_bfloat16, float);
  if (dtype == BN_BF16 && z_dtype == BN_BF16) GS_OUT(__nv_bfloat16, __nv_bfloat16);
#undef GS_OUT
  return BN_ERR_BAD_ARG;
}
