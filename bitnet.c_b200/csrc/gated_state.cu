// Recurrences of a matrix state per head under one decay per head and token: the gated delta rule and the
// state-space (Mamba-2) update, with the short convolutions in front of them and the gated norms behind.
//
// Per head, with a state S [dim, vdim] (float32, zero at a sequence's start, kept per slot), a log decay l_t and a
// factor b_t (both from per-head pre-activations):
//
//   delta rule     S' = e^l S;  u = b (v - S'^T k);  S = S' + k u^T;  o = S^T q       b = sigmoid(.),
//                  q and k unit vectors per head, q times a scale                     l = -e^A softplus(. + bias)
//   state space    S' = e^l S;  S = S' + b k v^T;    o = S^T q + D v                  b = softplus(. + bias), l = -e^A b
//                  (k: the input matrix B, q: the read-out C, v: the inner input x)
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
  const float* conv_w;        // [taps][channels]
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
      gs_load<float, V>(a.conv_w + (size_t)j * n_ch + c, w);
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
      float acc = fmaf(a.conv_w[(size_t)(a.taps - 1) * n_ch + c], x, a.conv_b ? a.conv_b[c] : 0.f);
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
  return a.proj && a.gate && a.conv_w && a.dt_bias && a.a_log && a.state && a.tok_seq && a.seq_start && a.seq_pos0 && a.slots &&
         a.groups > 0 && a.heads > 0 && a.heads % a.groups == 0 && a.dim > 0 && a.dim <= 256 && a.vdim > 0 && a.taps >= 1 &&
         a.taps <= GS_MAX_TAPS && a.q_off >= 0 && a.k_off >= 0 && a.v_off >= 0 && a.q_off + n_qk <= a.stride &&
         a.k_off + n_qk <= a.stride && a.v_off + n_v <= a.stride && a.a_off >= 0 && a.a_off + a.heads <= a.gate_stride &&
         a.b_off + a.heads <= a.gate_stride &&
         a.state_stride >= (size_t)a.heads * a.dim * a.vdim + (a.taps > 1 ? (size_t)a.taps * (2 * n_qk + n_v) : 0);
}

static GatedStateArgs gs_args(const void* proj, int n_tokens, int stride, int q_off, int k_off, int v_off, const float* gate,
                              int gate_stride, int a_off, int b_off, int groups, int heads, int dim, int vdim, int taps,
                              const float* conv_w, const float* conv_b, const float* dt_bias, const float* a_log, const float* d,
                              float q_scale, float* state, long long state_stride, const int* tok_seq, const int* seq_start,
                              const int* seq_pos0, const int* slots, int n_seqs) {
  GatedStateArgs a = {};
  a.proj = proj; a.gate = gate; a.conv_w = conv_w; a.conv_b = conv_b; a.dt_bias = dt_bias; a.a_log = a_log; a.d = d;
  a.state = state; a.tok_seq = tok_seq; a.seq_start = seq_start; a.seq_pos0 = seq_pos0; a.slots = slots;
  a.state_stride = (size_t)state_stride; a.q_scale = q_scale; a.stride = stride; a.gate_stride = gate_stride; a.q_off = q_off;
  a.k_off = k_off; a.v_off = v_off; a.a_off = a_off; a.b_off = b_off < 0 ? 0 : b_off; a.groups = groups; a.heads = heads; a.dim = dim;
  a.vdim = vdim; a.taps = taps; a.n_seqs = n_seqs; a.n_tokens = n_tokens;
  return a;
}

// The arguments all entry points share (b_off < 0: the state-space update, else the delta rule).
#define GS_PARAMS                                                                                                              \
  const void *proj, int dtype, int n_tokens, int stride, int q_off, int k_off, int v_off, const float *gate, int gate_stride,  \
      int a_off, int b_off, int groups, int heads, int dim, int vdim, int taps, const float *conv_w, const float *conv_b,      \
      const float *dt_bias, const float *a_log, const float *d, float q_scale, float *state, long long state_stride,           \
      const int *tok_seq, const int *seq_start, const int *seq_pos0, const int *slots, int n_seqs
#define GS_PASS                                                                                                                \
  proj, n_tokens, stride, q_off, k_off, v_off, gate, gate_stride, a_off, b_off, groups, heads, dim, vdim, taps, conv_w, conv_b, \
      dt_bias, a_log, d, q_scale, state, state_stride, tok_seq, seq_start, seq_pos0, slots, n_seqs

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
//   gate last    out = o / sqrt(mean over the part (o^2) + eps) * gain * silu(z)
// gain holds one number per place of the row, or per place of a part (gain_len = len: shared by the parts).
// THREADS 32: a warp per part, eight parts per block; else a block per part.  The part waits in shared memory.
template <typename T, typename G, int THREADS, int V>
__global__ void state_output_kernel(const float* __restrict__ o, const G* __restrict__ z, int z_stride, const float* __restrict__ gain,
                                    int gain_len, int parts, int len, float eps, int gate_first, T* __restrict__ out, int n_items) {
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
      if (!gate_first) w[e] *= gs_silu(g[e]);
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
                               float eps, int gate_first, void* out, int n_items, cudaStream_t stream) {
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
            eps, gate_first, (T*)out, n_items);
  return BN_OK;
}

extern "C" int bn_state_output(const float* o, const void* z, int z_dtype, int z_stride, const float* gain, int gain_len, int dtype,
                               int n_tokens, int parts, int len, float eps, int gate_first, void* out, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  if (!o || !z || !gain || !out || parts <= 0 || len <= 0 || z_stride < parts * len || !(eps > 0.f) ||
      (gain_len != len && gain_len != parts * len))
    return BN_ERR_BAD_ARG;
  const int items = n_tokens * parts;
  const bool vec = len % 4 == 0 && z_stride % 4 == 0 && !(((uintptr_t)o | (uintptr_t)z | (uintptr_t)gain | (uintptr_t)out) & 15);
#define GS_OUT(TT, GG)                                                                                                               \
  do {                                                                                                                               \
    if (len <= 512)                                                                                                                  \
      return vec ? launch_state_output<TT, GG, 32, 4>(o, z, z_stride, gain, gain_len, parts, len, eps, gate_first, out, items, stream) \
                 : launch_state_output<TT, GG, 32, 1>(o, z, z_stride, gain, gain_len, parts, len, eps, gate_first, out, items, stream); \
    return vec ? launch_state_output<TT, GG, 256, 4>(o, z, z_stride, gain, gain_len, parts, len, eps, gate_first, out, items, stream) \
               : launch_state_output<TT, GG, 256, 1>(o, z, z_stride, gain, gain_len, parts, len, eps, gate_first, out, items, stream); \
  } while (0)
  if (dtype == BN_F32 && z_dtype == BN_F32) GS_OUT(float, float);
  if (dtype == BN_BF16 && z_dtype == BN_F32) GS_OUT(__nv_bfloat16, float);
  if (dtype == BN_BF16 && z_dtype == BN_BF16) GS_OUT(__nv_bfloat16, __nv_bfloat16);
#undef GS_OUT
  return BN_ERR_BAD_ARG;
}
