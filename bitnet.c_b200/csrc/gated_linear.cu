// Gated linear recurrence per channel (the real-gated linear recurrent unit), with the short convolution in front of it and
// the gated read-out behind.
//
//   u_t = conv(x)_t + bias            a causal convolution per channel; the last tap is the current token's
//   r_t = sigmoid(R u_t + r_bias),  i_t = sigmoid(I u_t + i_bias)       R, I block-diagonal: `blocks` square parts
//   l_t = -8 r_t softplus(lam);  S_t = e^{l_t} S_{t-1} + sqrt(1 - e^{2 l_t}) i_t u_t;  out_t = scale * gelu_tanh(y_t) S_t
//
// x and y come as columns of the rows of a projection in the compute type; u is rounded to the compute type, everything
// behind it (gates, decays, states) is float32.
//
// Per-slot state, float32: [width] the recurrence's state, then (taps > 1) a ring of the convolution's inputs, [taps][width]:
// the input of position p lies in row p % taps.  A step of one token reads the rows of the taps - 1 positions before it
// and writes its own, which none of its readers asks for.
//
//   bn_gated_linear_token   one token per sequence: convolution, both gates, recurrence and read-out in one launch
//   bn_gated_linear_conv    runs of tokens: u [T, width]
//   bn_gated_linear_scan    runs of tokens, behind the gates' product: three launches.  Runs are cut into pieces of 64
//                           tokens; a first kernel takes every piece from a state of zero (its sum of log decays and its end
//                           state), a second carries the sequences' states through their pieces, a third takes every piece
//                           again from its true state, writes the outputs, and keeps state and ring.
#include "common.cuh"

#define GL_MAX_TAPS 16
#define GL_PIECE 64   // tokens per piece: the step's runs of new tokens
#define GL_THREADS 128

struct GatedLinearArgs {
  const void* x;            // [tokens, stride]: the convolution's inputs (first of `width` columns)
  const void* y;            // [tokens, stride]: the gate of the output
  int stride;
  const float* conv_w;      // [taps][width]
  const float* conv_b;      // [width]
  const float* gate_b;      // [blocks][2 wb]: the biases of r, then of i, part by part
  const float* lam;         // [width]
  float* state;
  size_t state_stride;
  int width, blocks, taps;
  const int* tok_seq;
  const int* seq_start;
  const int* seq_pos0;
  const int* slots;
  int n_seqs, n_tokens;
  float scale;
  void* out;                // [tokens, out_stride]: `width` columns, then `tail` columns: 1, 1, 0, 0, ...
  int out_stride, tail;
  __device__ __forceinline__ float* own(int s) const { return state + (size_t)slots[s] * state_stride; }
  __device__ __forceinline__ float* ring(int s) const { return own(s) + width; }
};

__device__ __forceinline__ float gl_sigmoid(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }
__device__ __forceinline__ float gl_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// (log decay, what enters the state) from the gates' pre-activations; sp = softplus(lam)
__device__ __forceinline__ float2 gl_step(float zr, float zi, float u, float sp) {
  const float l = -8.0f * gl_sigmoid(zr) * sp;
  return make_float2(l, sqrtf(-expm1f(2.0f * l)) * gl_sigmoid(zi) * u);
}

// ---- runs of tokens -------------------------------------------------------------------------------------
// A block takes a piece of a run and GL_CONV_COLS * V channels; a thread four neighbouring tokens of V neighbouring channels, so
// that a row is read once for the (up to) four outputs that look at it.
#define GL_CONV_COLS 16
#define GL_CONV_ROWS 4
template <typename T, int V>
__device__ __forceinline__ void gl_load(const T* p, float* o) {
  if constexpr (V * sizeof(T) == 16) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const T* v = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = to_f32<T>(v[e]);
  } else {
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = to_f32<T>(p[e]);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(GL_CONV_COLS * GL_PIECE / GL_CONV_ROWS)
gated_linear_conv_kernel(const GatedLinearArgs a, const int* __restrict__ tile_seq, const int* __restrict__ tile_row0, T* __restrict__ u) {
  pdl_launch_dependents();
  __shared__ __align__(16) float w[GL_MAX_TAPS][GL_CONV_COLS * V];
  const int c_block = blockIdx.y * GL_CONV_COLS * V;
  for (int i = threadIdx.x; i < a.taps * GL_CONV_COLS * V; i += blockDim.x) {
    const int j = i / (GL_CONV_COLS * V), d = i - j * GL_CONV_COLS * V;
    w[j][d] = c_block + d < a.width ? a.conv_w[(size_t)j * a.width + c_block + d] : 0.f;
  }
  __syncthreads();
  pdl_wait();
  const int s = tile_seq[blockIdx.x], start = a.seq_start[s], n = a.seq_start[s + 1] - start, pos0 = a.seq_pos0[s];
  const int d = (threadIdx.x % GL_CONV_COLS) * V, c = c_block + d;
  const int r0 = tile_row0[blockIdx.x] + threadIdx.x / GL_CONV_COLS * GL_CONV_ROWS;  // the thread's first row of the run
  if (c >= a.width || r0 >= n) return;
  const T* x = (const T*)a.x;
  const float* ring = a.ring(s);
  float acc[GL_CONV_ROWS][V];
#pragma unroll
  for (int o = 0; o < GL_CONV_ROWS; ++o)
#pragma unroll
    for (int e = 0; e < V; ++e) acc[o][e] = a.conv_b[c + e];
#pragma unroll 4
  for (int i = 1 - a.taps; i < GL_CONV_ROWS; ++i) {
    const int r = r0 + i;
    if (r >= n || pos0 + r < 0) continue;  // behind the run, or before the sequence
    float xv[V];
    if (r >= 0) gl_load<T, V>(x + (size_t)(start + r) * a.stride + c, xv);
    else gl_load<float, V>(ring + (size_t)((pos0 + r) % a.taps) * a.width + c, xv);
#pragma unroll
    for (int o = 0; o < GL_CONV_ROWS; ++o) {
      const int j = a.taps - 1 - (o - i);  // the tap of output o that looks at this row
      if (o >= i && j >= 0) {
#pragma unroll
        for (int e = 0; e < V; ++e) acc[o][e] = fmaf(w[j][d + e], xv[e], acc[o][e]);
      }
    }
  }
#pragma unroll
  for (int o = 0; o < GL_CONV_ROWS; ++o) {
    if (r0 + o >= n) break;
    T* dst = u + (size_t)(start + r0 + o) * a.width + c;
    if constexpr (V * sizeof(T) == 16) {
      uint4 raw;
      T* v = reinterpret_cast<T*>(&raw);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = from_f32<T>(acc[o][e]);
      *reinterpret_cast<uint4*>(dst) = raw;
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) dst[e] = from_f32<T>(acc[o][e]);
    }
  }
}

// A piece of a run and a channel per thread.  gates: [blocks][tokens][2 wb] float32.  OUT false: from a state of zero to the
// piece's sum of log decays and end state, piece_sums [pieces][2][width].  OUT true: from the state at
// piece_sums[.][1], to the outputs; the last piece of a sequence keeps the end state and the ring.
template <typename T, bool OUT>
__global__ void __launch_bounds__(GL_THREADS) gated_linear_piece_kernel(const GatedLinearArgs a, const T* __restrict__ u,
                                                                        const float* __restrict__ gates,
                                                                        const int* __restrict__ tile_seq, const int* __restrict__ tile_row0,
                                                                        float* __restrict__ piece_sums) {
  pdl_launch_dependents();
  pdl_wait();
  const int piece = blockIdx.x, c = blockIdx.y * GL_THREADS + threadIdx.x;
  const int s = tile_seq[piece], row0 = tile_row0[piece];
  const int start = a.seq_start[s], n = a.seq_start[s + 1] - start;
  const int first = start + row0, n_tok = min(GL_PIECE, n - row0);
  T* out = (T*)a.out;
  if (OUT && a.tail > 0 && blockIdx.y == 0) {
    for (int i = threadIdx.x; i < n_tok * a.tail; i += GL_THREADS) {
      const int t = i / a.tail, j = i - t * a.tail;
      out[(size_t)(first + t) * a.out_stride + a.width + j] = from_f32<T>(j < 2 ? 1.0f : 0.f);
    }
  }
  if (c >= a.width) return;
  const int wb = a.width / a.blocks, b = c / wb, d = c - b * wb;
  const float* g = gates + ((size_t)b * a.n_tokens + first) * 2 * wb + d;
  const float br = a.gate_b[(size_t)b * 2 * wb + d], bi = a.gate_b[(size_t)b * 2 * wb + wb + d];
  const float sp = gl_softplus(a.lam[c]);
  const T* ut = u + (size_t)first * a.width + c;
  const T* yt = (const T*)a.y + (size_t)first * a.stride + c;
  float* mine = piece_sums + (size_t)piece * 2 * a.width + c;
  float S = OUT ? mine[a.width] : 0.f, L = 0.f;
  // eight tokens at a time, the next eight on their way meanwhile
  constexpr int B = 8;
  float zr[2][B], zi[2][B], uu[2][B], yy[2][B];
  auto fetch = [&](int t0, int buf) {
#pragma unroll
    for (int e = 0; e < B; ++e) {
      const int t = min(t0 + e, n_tok - 1);
      zr[buf][e] = g[(size_t)t * 2 * wb];
      zi[buf][e] = g[(size_t)t * 2 * wb + wb];
      uu[buf][e] = to_f32<T>(ut[(size_t)t * a.width]);
      yy[buf][e] = OUT ? to_f32<T>(yt[(size_t)t * a.stride]) : 0.f;
    }
  };
  fetch(0, 0);
  for (int t2 = 0; t2 < n_tok; t2 += 2 * B) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t0 = t2 + half * B;
      if (t0 + B < n_tok) fetch(t0 + B, half ^ 1);
#pragma unroll
      for (int e = 0; e < B; ++e) {
        if (t0 + e < n_tok) {
          const float2 st = gl_step(zr[half][e] + br, zi[half][e] + bi, uu[half][e], sp);
          S = fmaf(expf(st.x), S, st.y);
          if (OUT)
            out[(size_t)(first + t0 + e) * a.out_stride + c] = from_f32<T>(a.scale * glu_activation(yy[half][e], BN_ACT_GELU_TANH) * S);
          else
            L += st.x;
        }
      }
    }
  }
  if (!OUT) {
    mine[0] = L;
    mine[a.width] = S;
  } else if (row0 + n_tok == n) {
    a.own(s)[c] = S;
    if (a.taps > 1) {
      float* ring = a.ring(s);
      const int pos0 = a.seq_pos0[s];
      const T* x = (const T*)a.x;
      for (int r = max(0, n - (a.taps - 1)); r < n; ++r)
        ring[(size_t)((pos0 + r) % a.taps) * a.width + c] = to_f32<T>(x[(size_t)(start + r) * a.stride + c]);
    }
  }
}

// A sequence and a channel per thread: piece_sums[.][1] becomes the state before the piece.
__global__ void __launch_bounds__(GL_THREADS) gated_linear_carry_kernel(const GatedLinearArgs a, const int* __restrict__ tile_seq,
                                                                        const int* __restrict__ tile_row0, int n_pieces,
                                                                        float* __restrict__ piece_sums) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ int order[];  // the sequence's pieces by their row
  const int s = blockIdx.x, c = blockIdx.y * GL_THREADS + threadIdx.x;
  const int n = a.seq_start[s + 1] - a.seq_start[s], count = (n + GL_PIECE - 1) / GL_PIECE;
  for (int i = threadIdx.x; i < n_pieces; i += GL_THREADS)
    if (tile_seq[i] == s) order[tile_row0[i] / GL_PIECE] = i;
  __syncthreads();
  if (c >= a.width) return;
  float S = a.own(s)[c];
  constexpr int B = 8;
  for (int p0 = 0; p0 < count; p0 += B) {
    float L[B], E[B];
#pragma unroll
    for (int e = 0; e < B; ++e) {
      const float* p = piece_sums + (size_t)order[min(p0 + e, count - 1)] * 2 * a.width + c;
      L[e] = p[0];
      E[e] = p[a.width];
    }
#pragma unroll
    for (int e = 0; e < B; ++e)
      if (p0 + e < count) {
        piece_sums[(size_t)order[p0 + e] * 2 * a.width + a.width + c] = S;
        S = fmaf(expf(L[e]), S, E[e]);
      }
  }
}

// ---- one token per sequence --------------------------------------------------------------------------------
#define GL_SEQS 8        // sequences a block takes at a time
#define GL_CHANNELS 8    // channels a block takes at a time: one per warp
#define GL_TOKEN_BLOCKS 300  // about two blocks per SM: every block convolves its whole part
#define GL_AHEAD 8       // numbers of each row of R and I that a lane asks for before the step's inputs are there

// Blocks share out a part's channels eight at a time: the convolution of the whole part for eight sequences at a time into
// shared memory, then a warp per channel takes its rows of R and I (w_gates [blocks][2 wb][wb], r's rows first) against all of them, and
// lane s does sequence s's step.
// TAPS: the most taps the instantiation takes (their loads are all in flight together).
template <typename T, int TAPS>
__global__ void __launch_bounds__(256) gated_linear_token_kernel(const GatedLinearArgs a, const T* __restrict__ w_gates) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float us[];  // [GL_SEQS][wb padded to 4]
  __shared__ int seq_pos[GL_SEQS], seq_row[GL_SEQS];
  __shared__ float* seq_own[GL_SEQS];
  const int wb = a.width / a.blocks, ld = (wb + 3) / 4 * 4;
  const int b = blockIdx.x, first = blockIdx.y * GL_CHANNELS, step = gridDim.y * GL_CHANNELS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const T* x = (const T*)a.x;
  T* out = (T*)a.out;
  // what of the warp's first channel are weights
  float wr[GL_AHEAD], wi[GL_AHEAD], br = 0.f, bi = 0.f, sp = 0.f;
  auto weights_of = [&](int d) {
    const bool live = d < wb;
    const T* rr = w_gates + ((size_t)b * 2 * wb + (live ? d : 0)) * wb;
    const T* ri = rr + (size_t)wb * wb;
#pragma unroll
    for (int k = 0; k < GL_AHEAD; ++k) {
      const int jj = lane + 32 * k;
      wr[k] = jj < wb ? to_f32<T>(rr[jj]) : 0.f;
      wi[k] = jj < wb ? to_f32<T>(ri[jj]) : 0.f;
    }
    if (live) {
      br = a.gate_b[(size_t)b * 2 * wb + d];
      bi = a.gate_b[(size_t)b * 2 * wb + wb + d];
      sp = gl_softplus(a.lam[b * wb + d]);
    }
  };
  weights_of(first + warp);
  pdl_wait();
  if (a.tail > 0 && blockIdx.x == 0 && blockIdx.y == 0)
    for (int i = threadIdx.x; i < a.n_seqs * a.tail; i += blockDim.x) {
      const int s = i / a.tail, j = i - s * a.tail;
      out[(size_t)s * a.out_stride + a.width + j] = from_f32<T>(j < 2 ? 1.0f : 0.f);
    }
  for (int s0 = 0; s0 < a.n_seqs; s0 += GL_SEQS) {
    const int ns = min(GL_SEQS, a.n_seqs - s0);
    __syncthreads();  // the sequences before are done with the inputs
    if (threadIdx.x < ns) {
      const int s = s0 + threadIdx.x;
      seq_pos[threadIdx.x] = a.seq_pos0[s];
      seq_row[threadIdx.x] = a.seq_start[s];
      seq_own[threadIdx.x] = a.own(s);
    }
    __syncthreads();
    // lane s: sequence s's state and output gate, on their way during the convolution (of the next channel: during this one's
    // sums)
    float S_next = 0.f, y_next = 0.f;
    auto inputs_of = [&](int d) {
      if (d < wb && lane < ns) {
        S_next = seq_own[lane][b * wb + d];
        y_next = to_f32<T>(((const T*)a.y)[(size_t)seq_row[lane] * a.stride + b * wb + d]);
      }
    };
    inputs_of(first + warp);
#pragma unroll (TAPS <= 4 ? 4 : 1)
    for (int i = threadIdx.x; i < GL_SEQS * ld; i += blockDim.x) {
      const int q = i / ld, dd = i - q * ld;
      float acc = 0.f;
      if (q < ns && dd < wb) {
        const int pos = seq_pos[q], cc = b * wb + dd;
        float* ring = seq_own[q] + a.width;
        const float now = to_f32<T>(x[(size_t)seq_row[q] * a.stride + cc]);
        acc = fmaf(a.conv_w[(size_t)(a.taps - 1) * a.width + cc], now, a.conv_b[cc]);
        int row = pos % a.taps;  // of this token; the token `back` before it lies `back` rows in front
        if (a.taps > 1 && dd / GL_CHANNELS % gridDim.y == blockIdx.y) ring[(size_t)row * a.width + cc] = now;
        float before[TAPS], w[TAPS];
#pragma unroll
        for (int back = 1; back < TAPS; ++back) {
          row = row == 0 ? a.taps - 1 : row - 1;
          const bool there = back < a.taps && back <= pos;
          before[back] = there ? ring[(size_t)row * a.width + cc] : 0.f;
          w[back] = there ? a.conv_w[(size_t)(a.taps - 1 - back) * a.width + cc] : 0.f;
        }
#pragma unroll
        for (int back = 1; back < TAPS; ++back) acc = fmaf(w[back], before[back], acc);
        acc = to_f32<T>(from_f32<T>(acc));
      }
      us[i] = acc;
    }
    __syncthreads();
    for (int d = first + warp; d < wb; d += step) {
      const int c = b * wb + d;
      const T* rr = w_gates + ((size_t)b * 2 * wb + d) * wb;
      const T* ri = rr + (size_t)wb * wb;
      const float S_old = S_next, y = y_next;
      float zr[GL_SEQS], zi[GL_SEQS];
#pragma unroll
      for (int q = 0; q < GL_SEQS; ++q) zr[q] = zi[q] = 0.f;
#pragma unroll
      for (int k = 0; k < GL_AHEAD; ++k) {
        const int j = lane + 32 * k;
        if (j < wb) {
#pragma unroll
          for (int q = 0; q < GL_SEQS; ++q) {
            const float v = us[q * ld + j];
            zr[q] = fmaf(wr[k], v, zr[q]);
            zi[q] = fmaf(wi[k], v, zi[q]);
          }
        }
      }
      for (int j = lane + 32 * GL_AHEAD; j < wb; j += 32) {
        const float vr = to_f32<T>(rr[j]), vi = to_f32<T>(ri[j]);
#pragma unroll
        for (int q = 0; q < GL_SEQS; ++q) {
          const float v = us[q * ld + j];
          zr[q] = fmaf(vr, v, zr[q]);
          zi[q] = fmaf(vi, v, zi[q]);
        }
      }
      const float my_br = br, my_bi = bi, my_sp = sp;
      // this channel's weights have been used: the next one's, or the first one's for the next sequences
      const int next = d + step < wb ? d + step : first + warp;
      if (next != d) {
        weights_of(next);
        if (next > d) inputs_of(next);
      }
      float my_r = 0.f, my_i = 0.f;
#pragma unroll
      for (int q = 0; q < GL_SEQS; ++q) {
        const float r = warp_sum(zr[q]), i = warp_sum(zi[q]);
        if (lane == q) { my_r = r; my_i = i; }
      }
      if (lane < ns) {
        const float2 st = gl_step(my_r + my_br, my_i + my_bi, us[lane * ld + d], my_sp);
        const float S = fmaf(expf(st.x), S_old, st.y);
        seq_own[lane][c] = S;
        out[(size_t)seq_row[lane] * a.out_stride + c] = from_f32<T>(a.scale * glu_activation(y, BN_ACT_GELU_TANH) * S);
      }
    }
  }
}

static bool gl_fits(const GatedLinearArgs& a) {
  return a.x && a.y && a.conv_w && a.conv_b && a.gate_b && a.lam && a.state && a.tok_seq && a.seq_start && a.seq_pos0 && a.slots &&
         a.width > 0 && a.blocks > 0 && a.width % a.blocks == 0 && a.taps >= 1 && a.taps <= GL_MAX_TAPS && a.stride >= a.width &&
         a.tail >= 0 && a.n_seqs > 0 && a.state_stride >= (size_t)a.width * (1 + (a.taps > 1 ? a.taps : 0));
}

// The arguments all entry points share.
#define GL_PARAMS                                                                                                                 \
  const void *x, const void *y, int dtype, int n_tokens, int stride, int width, int blocks, int taps, const float *conv_w,        \
      const float *conv_b, const float *gate_b, const float *lam, float *state, long long state_stride, const int *tok_seq,       \
      const int *seq_start, const int *seq_pos0, const int *slots, int n_seqs, float scale, void *out, int out_stride, int tail
static GatedLinearArgs gl_args(GL_PARAMS) {
  (void)dtype;
  GatedLinearArgs a = {};
  a.x = x; a.y = y; a.stride = stride; a.conv_w = conv_w; a.conv_b = conv_b; a.gate_b = gate_b; a.lam = lam; a.state = state;
  a.state_stride = (size_t)state_stride; a.width = width; a.blocks = blocks; a.taps = taps; a.tok_seq = tok_seq;
  a.seq_start = seq_start; a.seq_pos0 = seq_pos0; a.slots = slots; a.n_seqs = n_seqs; a.n_tokens = n_tokens; a.scale = scale;
  a.out = out; a.out_stride = out_stride; a.tail = tail;
  return a;
}
#define GL_PASS                                                                                                                \
  x, y, dtype, n_tokens, stride, width, blocks, taps, conv_w, conv_b, gate_b, lam, state, state_stride, tok_seq, seq_start, seq_pos0, \
      slots, n_seqs, scale, out, out_stride, tail

// u [n_tokens, width] in the compute type; tile_seq / tile_row0: the sequence and first row of every piece of 64 new tokens.
extern "C" int bn_gated_linear_conv(GL_PARAMS, const int* tile_seq, const int* tile_row0, int n_pieces, void* u, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  const GatedLinearArgs a = gl_args(GL_PASS);
  if (!gl_fits(a) || !u || !tile_seq || !tile_row0 || n_pieces <= 0) return BN_ERR_BAD_ARG;
#define GL_CONV(TT, VV)                                                                                                              \
  do {                                                                                                                               \
    const int per = GL_CONV_COLS * VV, cols = (width + per - 1) / per;                                                               \
    if (cols > 65535) return BN_ERR_BAD_ARG;                                                                                         \
    BN_LAUNCH((gated_linear_conv_kernel<TT, VV>), dim3(n_pieces, cols), GL_CONV_COLS * GL_PIECE / GL_CONV_ROWS, 0, stream, a, tile_seq, \
              tile_row0, (TT*)u);                                                                                                    \
  } while (0)
  const int v = dtype == BN_F32 ? 4 : 8;  // whole 16-byte pieces, also of the ring's rows
  const bool vec = width % v == 0 && stride % v == 0 && state_stride % 4 == 0 && !(((uintptr_t)x | (uintptr_t)u | (uintptr_t)state) & 15);
  if (dtype == BN_F32) { if (vec) GL_CONV(float, 4); else GL_CONV(float, 1); }
  else if (dtype == BN_BF16) { if (vec) GL_CONV(__nv_bfloat16, 8); else GL_CONV(__nv_bfloat16, 1); }
  else return BN_ERR_BAD_ARG;
#undef GL_CONV
  return BN_OK;
}

// gates [blocks][n_tokens][2 width / blocks]: the products R u and I u without their biases; tile_seq / tile_row0: the sequence and
// first row of every piece of 64 new tokens; piece_sums [n_pieces][2][width]: working space.
extern "C" int bn_gated_linear_scan(GL_PARAMS, const void* u, const float* gates, const int* tile_seq, const int* tile_row0, int n_pieces,
                                    float* piece_sums, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  const GatedLinearArgs a = gl_args(GL_PASS);
  const size_t smem = (size_t)n_pieces * sizeof(int);
  const int cols = (width + GL_THREADS - 1) / GL_THREADS;
  if (!gl_fits(a) || !u || !gates || !tile_seq || !tile_row0 || n_pieces <= 0 || !piece_sums || !out || out_stride < width + tail ||
      smem > 200 * 1024 || cols > 65535)
    return BN_ERR_BAD_ARG;
  static size_t granted = 0;
  if (smem > 48 * 1024 && smem > granted) {
    cudaError_t e = cudaFuncSetAttribute(gated_linear_carry_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return BN_ERR_LAUNCH + (int)e;
    granted = smem;
  }
  const dim3 pieces(n_pieces, cols);
#define GL_RUN(TT)                                                                                                                    \
  do {                                                                                                                                \
    BN_LAUNCH((gated_linear_piece_kernel<TT, false>), pieces, GL_THREADS, 0, stream, a, (const TT*)u, gates, tile_seq, tile_row0, piece_sums); \
    BN_LAUNCH(gated_linear_carry_kernel, dim3(n_seqs, cols), GL_THREADS, smem, stream, a, tile_seq, tile_row0, n_pieces, piece_sums); \
    BN_LAUNCH((gated_linear_piece_kernel<TT, true>), pieces, GL_THREADS, 0, stream, a, (const TT*)u, gates, tile_seq, tile_row0, piece_sums); \
  } while (0)
  if (dtype == BN_F32) GL_RUN(float);
  else if (dtype == BN_BF16) GL_RUN(__nv_bfloat16);
  else return BN_ERR_BAD_ARG;
#undef GL_RUN
  return BN_OK;
}

// w_gates [blocks][2 wb][wb] in the compute type: R's rows, then I's, part by part.
extern "C" int bn_gated_linear_token(GL_PARAMS, const void* w_gates, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  const GatedLinearArgs a = gl_args(GL_PASS);
  if (!gl_fits(a) || !w_gates || !out || out_stride < width + tail || n_tokens != n_seqs) return BN_ERR_BAD_ARG;
  const int wb = width / blocks;
  const size_t smem = (size_t)GL_SEQS * ((wb + 3) / 4 * 4) * sizeof(float);
  const int groups = (wb + GL_CHANNELS - 1) / GL_CHANNELS, want = (GL_TOKEN_BLOCKS + blocks - 1) / blocks;
  const dim3 grid(blocks, groups < want ? groups : want);
  if (smem > 200 * 1024) return BN_ERR_BAD_ARG;
#define GL_TOKEN(TT, NN)                                                                                                               \
  do {                                                                                                                                 \
    static size_t granted = 0;                                                                                                         \
    if (smem > 48 * 1024 && smem > granted) {                                                                                          \
      cudaError_t e = cudaFuncSetAttribute(gated_linear_token_kernel<TT, NN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (e != cudaSuccess) return BN_ERR_LAUNCH + (int)e;                                                                             \
      granted = smem;                                                                                                                  \
    }                                                                                                                                  \
    BN_LAUNCH((gated_linear_token_kernel<TT, NN>), grid, 256, smem, stream, a, (const TT*)w_gates);                                    \
  } while (0)
  if (dtype == BN_F32) { if (taps <= 4) GL_TOKEN(float, 4); else GL_TOKEN(float, GL_MAX_TAPS); }
  else if (dtype == BN_BF16) { if (taps <= 4) GL_TOKEN(__nv_bfloat16, 4); else GL_TOKEN(__nv_bfloat16, GL_MAX_TAPS); }
  else return BN_ERR_BAD_ARG;
#undef GL_TOKEN
  return BN_OK;
}
