// A residual carried in several streams, the layer norm that reads it, and the causal convolution that a
// sublayer adds to its normed input.
//
// x [rows, streams * width] float32: row r holds its streams one behind another.  One pass over a row does
//
//   X <- M^T X + mult * out (scale * y)^T       (X: the streams as rows; left out without y)
//   u = read^T X                                (read null: the rows' plain sum)
//   h = (u - mean(u)) / sqrt(var(u) + eps) * w + b
//
// with y the delta of the sublayer that ran before (any type), `scale` one number per channel.  Without mix (and
// with one stream) it is an ordinary residual sum and a layer norm.  With a row index only the listed rows are read
// and written densely, and x stays as it is (the final norm).  Sums and statistics are float32; the variance is
// taken around the mean in a second pass over the row's numbers on the chip.
//
// The input convolution: h'_t = h_t + sum_j taps[j] h_(t - n + 1 + j) per channel, with zeros where a sequence has no input yet.
// h is what the compute type holds, so that a sequence's last n - 1 inputs, kept per slot in that type
// (hist [slots, n - 1, width], oldest first), are the same numbers whether they came from this step or an earlier
// one.  Steps of one token per sequence take it inside the norm's pass (a thread owns its columns: it reads the
// history, shifts it and adds the new input); steps with runs of tokens in a pass of its own over the normed rows.
#include "common.cuh"
#include <cooperative_groups.h>
namespace cg = cooperative_groups;

#define ST_MAX_STREAMS 16
#define ST_CLUSTER 8
#define ST_MAX_TAPS 16

struct StreamsArgs {
  float* x;
  const void* y;          // null: no update
  const float* mix;       // [streams][streams] (from, to) and then out [streams]; null: identity and ones
  const float* scale;     // [width] or null
  const float* read;      // [streams] or null
  const void* w;
  const void* b;          // null: none
  const int* rows;        // null: every row
  void* out;
  const float* taps;      // [n_taps][width] or null
  void* hist;             // [slots, hist_stride] in the output's type
  const int* slots;       // slot of row r (steps of one token per sequence)
  size_t hist_stride;
  float mult, eps;
  int y_dtype, w_dtype, b_dtype, out_dtype, width, streams, n_taps, cols, write_x;
};

template <int V>
__device__ __forceinline__ void load_v(const void* p, int dtype, size_t i, float* o) {
  if (V == 4) {
    if (dtype == BN_F32) {
      const float4 a = *reinterpret_cast<const float4*>((const float*)p + i);
      o[0] = a.x; o[1 % V] = a.y; o[2 % V] = a.z; o[3 % V] = a.w;
    } else {
      const uint2 raw = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)p + i);
      const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
      const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
      o[0] = a.x; o[1 % V] = a.y; o[2 % V] = b.x; o[3 % V] = b.y;
    }
  } else {
    o[0] = load_as_f32(p, dtype, i);
  }
}
template <int V>
__device__ __forceinline__ void store_v(void* p, int dtype, size_t i, const float* v) {
  if (V == 4) {
    if (dtype == BN_F32) {
      *reinterpret_cast<float4*>((float*)p + i) = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]);
    } else {
      const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1 % V]), b = __floats2bfloat162_rn(v[2 % V], v[3 % V]);
      uint2 raw;
      raw.x = *reinterpret_cast<const unsigned*>(&a);
      raw.y = *reinterpret_cast<const unsigned*>(&b);
      *reinterpret_cast<uint2*>((__nv_bfloat16*)p + i) = raw;
    }
  } else {
    store_from_f32(p, dtype, i, v[0]);
  }
}

// A block takes the columns [rank * cols, (rank + 1) * cols) of a row (rank 0 and the whole row without a cluster).
// MS: room for so many streams in registers.  V: columns a thread takes at once.
template <int MS, int V, bool CL>
__global__ void streams_norm_kernel(const StreamsArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float u_row[];  // cols
  __shared__ float scratch[32];
  __shared__ float part[2];
  __shared__ float coef[MS * MS + 2 * MS];  // mix, out, read
  const int S = a.streams, width = a.width;
  for (int i = threadIdx.x; i < S * S + S; i += blockDim.x) coef[i] = a.mix ? a.mix[i] : 1.0f;  // without mix there is one stream
  for (int i = threadIdx.x; i < S; i += blockDim.x) coef[S * S + S + i] = a.read ? a.read[i] : 1.0f;
  pdl_wait();
  __syncthreads();
  const int r = blockIdx.x, rank = CL ? blockIdx.y : 0;
  const size_t row = a.rows ? (size_t)a.rows[r] : (size_t)r;
  float* xr = a.x + row * (size_t)S * width;
  const int c0 = rank * a.cols, c1 = min(width, c0 + a.cols);
  float sum = 0.f;
  for (int c = c0 + threadIdx.x * V; c < c1; c += blockDim.x * V) {
    float xs[MS][V], u[V];
#pragma unroll
    for (int s = 0; s < MS; ++s)
      if (s < S) load_v<V>(xr, BN_F32, (size_t)s * width + c, xs[s]);
#pragma unroll
    for (int e = 0; e < V; ++e) u[e] = 0.f;
    if (a.y) {
      float y[V];
      load_v<V>(a.y, a.y_dtype, row * width + c, y);
      if (a.scale) {
        float sc[V];
        load_v<V>(a.scale, BN_F32, c, sc);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] *= sc[e];
      }
#pragma unroll
      for (int t = 0; t < MS; ++t) {
        if (t < S) {
          float v[V];
          const float k = a.mult * coef[S * S + t];
#pragma unroll
          for (int e = 0; e < V; ++e) v[e] = 0.f;
#pragma unroll
          for (int s = 0; s < MS; ++s)
            if (s < S) {
              const float m = coef[s * S + t];
#pragma unroll
              for (int e = 0; e < V; ++e) v[e] = fmaf(m, xs[s][e], v[e]);
            }
          const float rd = coef[S * S + S + t];
#pragma unroll
          for (int e = 0; e < V; ++e) {
            v[e] = fmaf(k, y[e], v[e]);
            u[e] = fmaf(rd, v[e], u[e]);
          }
          if (a.write_x) store_v<V>(xr, BN_F32, (size_t)t * width + c, v);  // this thread has read all its columns' streams
        }
      }
    } else {
#pragma unroll
      for (int s = 0; s < MS; ++s)
        if (s < S) {
          const float rd = coef[S * S + S + s];
#pragma unroll
          for (int e = 0; e < V; ++e) u[e] = fmaf(rd, xs[s][e], u[e]);
        }
    }
    store_v<V>(u_row, BN_F32, c - c0, u);
#pragma unroll
    for (int e = 0; e < V; ++e) sum += u[e];
  }
  sum = block_sum(sum, scratch);
  if (CL) {
    cg::cluster_group cluster = cg::this_cluster();
    if (threadIdx.x == 0) part[0] = sum;
    cluster.sync();
    sum = 0.f;
    for (int k = 0; k < ST_CLUSTER; ++k) sum += *cluster.map_shared_rank(&part[0], k);
  }
  const float mean = sum / (float)width;
  float ss = 0.f;
  for (int c = c0 + threadIdx.x * V; c < c1; c += blockDim.x * V) {
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float d = u_row[c - c0 + e] - mean;
      ss = fmaf(d, d, ss);
    }
  }
  ss = block_sum(ss, scratch);
  if (CL) {
    cg::cluster_group cluster = cg::this_cluster();
    if (threadIdx.x == 0) part[1] = ss;
    cluster.sync();
    ss = 0.f;
    for (int k = 0; k < ST_CLUSTER; ++k) ss += *cluster.map_shared_rank(&part[1], k);
  }
  const float inv = 1.0f / sqrtf(ss / (float)width + a.eps);
  const size_t hist0 = a.hist ? (size_t)a.slots[r] * a.hist_stride : 0;
  for (int c = c0 + threadIdx.x * V; c < c1; c += blockDim.x * V) {
    float h[V], w[V], b[V];
    load_v<V>(a.w, a.w_dtype, c, w);
    if (a.b) load_v<V>(a.b, a.b_dtype, c, b);
#pragma unroll
    for (int e = 0; e < V; ++e) h[e] = (u_row[c - c0 + e] - mean) * inv * w[e] + (a.b ? b[e] : 0.f);
    if (a.taps) {
      if (a.out_dtype == BN_BF16) {
#pragma unroll
        for (int e = 0; e < V; ++e) h[e] = __bfloat162float(__float2bfloat16_rn(h[e]));
      }
      float acc[V], t[V], v[V];
      load_v<V>(a.taps, BN_F32, (size_t)(a.n_taps - 1) * width + c, t);
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = t[e] * h[e];
      for (int j = 0; j < a.n_taps - 1; ++j) {  // history row j is the input n_taps - 1 - j positions back
        load_v<V>(a.hist, a.out_dtype, hist0 + (size_t)j * width + c, v);
        load_v<V>(a.taps, BN_F32, (size_t)j * width + c, t);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(t[e], v[e], acc[e]);
        if (j > 0) store_v<V>(a.hist, a.out_dtype, hist0 + (size_t)(j - 1) * width + c, v);
      }
      if (a.n_taps > 1) store_v<V>(a.hist, a.out_dtype, hist0 + (size_t)(a.n_taps - 2) * width + c, h);
#pragma unroll
      for (int e = 0; e < V; ++e) h[e] += acc[e];
    }
    store_v<V>(a.out, a.out_dtype, (size_t)r * width + c, h);
  }
  if (CL) cg::this_cluster().sync();  // no block may leave while another still reads its sums
}

template <int MS, int V>
static int launch_streams(const StreamsArgs& args, int n_rows, cudaStream_t stream) {
  StreamsArgs a = args;
  const bool cluster = V == 4 && n_rows <= 256 && a.width >= 1024;
  a.cols = cluster ? ((a.width + ST_CLUSTER - 1) / ST_CLUSTER + 3) / 4 * 4 : a.width;
  const size_t smem = (((size_t)a.cols + 3) / 4 * 4) * sizeof(float);
  if (smem > 200 * 1024) return BN_ERR_BAD_ARG;
  int threads = ((a.cols + V - 1) / V + 31) / 32 * 32;
  threads = min(threads, MS <= 4 ? 512 : 256);
  cudaError_t e;
  if (cluster) {
    if (smem > 48 * 1024) {
      static size_t granted = 0;
      if (smem > granted) {
        e = cudaFuncSetAttribute(streams_norm_kernel<MS, V, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return BN_ERR_LAUNCH + (int)e;
        granted = smem;
      }
    }
    e = bn_launch_cluster(streams_norm_kernel<MS, V, true>, dim3(n_rows, ST_CLUSTER), dim3(threads), smem, stream,
                          dim3(1, ST_CLUSTER, 1), a);
  } else {
    if (smem > 48 * 1024) {
      static size_t granted = 0;
      if (smem > granted) {
        e = cudaFuncSetAttribute(streams_norm_kernel<MS, V, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return BN_ERR_LAUNCH + (int)e;
        granted = smem;
      }
    }
    e = bn_launch(streams_norm_kernel<MS, V, false>, dim3(n_rows), dim3(threads), smem, stream, a);
  }
  return e == cudaSuccess ? BN_OK : BN_ERR_LAUNCH + (int)e;
}

// See the head of the file.  mix: [streams * streams] numbers (from, to), then the streams' out factors, or null.
// taps [n_taps, width] float32 with hist / slots: one token per sequence, row r belongs to slot slots[r].
extern "C" int bn_streams_norm(float* x, int n_rows, int width, int streams, const void* y, int y_dtype, const float* mix,
                               const float* scale, float mult, const float* read, const void* w, int w_dtype, const void* b,
                               int b_dtype, float eps, const int* rows, int write_x, void* out, int out_dtype,
                               const float* taps, int n_taps, void* hist, long long hist_stride, const int* slots,
                               cudaStream_t stream) {
  if (n_rows <= 0) return BN_OK;
  if (!x || !w || !out || width <= 0 || streams < 1 || streams > ST_MAX_STREAMS || !(eps > 0.f) || (streams > 1 && y && !mix) ||
      (rows && (write_x || taps)) || (taps && (n_taps < 1 || n_taps > ST_MAX_TAPS || (n_taps > 1 && (!hist || !slots)))))
    return BN_ERR_BAD_ARG;
  StreamsArgs a = {};
  a.x = x; a.y = y; a.mix = mix; a.scale = scale; a.read = read; a.w = w; a.b = b; a.rows = rows; a.out = out; a.taps = taps;
  a.hist = taps && n_taps > 1 ? hist : nullptr; a.slots = slots; a.hist_stride = (size_t)hist_stride; a.mult = mult; a.eps = eps;
  a.y_dtype = y_dtype; a.w_dtype = w_dtype; a.b_dtype = b_dtype; a.out_dtype = out_dtype; a.width = width; a.streams = streams;
  a.n_taps = n_taps; a.write_x = write_x && y;
  const bool vec = width % 8 == 0 && hist_stride % 8 == 0 &&
                   !(((uintptr_t)x | (uintptr_t)y | (uintptr_t)scale | (uintptr_t)w | (uintptr_t)b | (uintptr_t)out | (uintptr_t)taps |
                      (uintptr_t)hist) & 15);
  if (streams == 1) return vec ? launch_streams<1, 4>(a, n_rows, stream) : launch_streams<1, 1>(a, n_rows, stream);
  if (streams == 2) return vec ? launch_streams<2, 4>(a, n_rows, stream) : launch_streams<2, 1>(a, n_rows, stream);
  if (streams <= 4) return vec ? launch_streams<4, 4>(a, n_rows, stream) : launch_streams<4, 1>(a, n_rows, stream);
  if (streams <= 8) return vec ? launch_streams<8, 4>(a, n_rows, stream) : launch_streams<8, 1>(a, n_rows, stream);
  return launch_streams<16, 1>(a, n_rows, stream);
}

// Runs of tokens: out[t] = h[t] + sum_j taps[j] h[t - n_taps + 1 + j] over the rows of each sequence, inputs before the
// step from its slot's history, which then receives the last n_taps - 1 inputs.  The first n_taps - 1 rows of a sequence
// read the history: the thread that owns a column group of the first row takes all of these rows, one after another, and
// then replaces the history, so nobody else touches those columns of it.
template <typename T, int V>
__device__ __forceinline__ void convolve_first_rows(const T* h, T* out, int width, const float* taps, int n_taps, T* hs, int start, int n,
                                                    int c) {
  const int dtype = sizeof(T) == 4 ? BN_F32 : BN_BF16, back = n_taps - 1;
  for (int i = 0; i < min(n, back); ++i) {
    float acc[V], v[V], w[V];
    load_v<V>(h, dtype, (size_t)(start + i) * width + c, acc);
    for (int j = 0; j <= back; ++j) {
      const int src = i - back + j;  // place among the sequence's new rows
      if (src >= 0) load_v<V>(h, dtype, (size_t)(start + src) * width + c, v);
      else load_v<V>(hs, dtype, (size_t)(back + src) * width, v);
      load_v<V>(taps, BN_F32, (size_t)j * width + c, w);
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = fmaf(w[e], v[e], acc[e]);
    }
    store_v<V>(out, dtype, (size_t)(start + i) * width + c, acc);
  }
  for (int j = 0; j < back; ++j) {  // rising j: what is still needed lies ahead of what is overwritten
    float v[V];
    const int src = j + n;
    if (src < back) load_v<V>(hs, dtype, (size_t)src * width, v);
    else load_v<V>(h, dtype, (size_t)(start + src - back) * width + c, v);
    store_v<V>(hs, dtype, (size_t)j * width, v);
  }
}

// A thread takes V columns of R neighbouring packed rows; with N taps fixed the rows it looks at are read once and wait
// in registers (N 0: any number of taps, every input is read where it is needed).  Grid (column groups, row groups).
template <typename T, int V, int N, int R>
__global__ void __launch_bounds__(128) input_convolution_kernel(const T* __restrict__ h, T* __restrict__ out, int width, int n_tokens,
                                                                const float* __restrict__ taps, int n_taps, T* hist, size_t hist_stride,
                                                                const int* __restrict__ tok_seq, const int* __restrict__ seq_start,
                                                                const int* __restrict__ slots) {
  pdl_launch_dependents();
  const int dtype = sizeof(T) == 4 ? BN_F32 : BN_BF16;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V, t0 = blockIdx.y * R;
  if (c >= width) return;
  const int back = (N ? N : n_taps) - 1;
  float w[N ? N : 1][V];
  if (N) {
#pragma unroll
    for (int j = 0; j < N; ++j) load_v<V>(taps, BN_F32, (size_t)j * width + c, w[j]);
  }
  pdl_wait();
  float x[N ? R + N - 1 : 1][V];
  if (N) {
#pragma unroll
    for (int i = 0; i < R + N - 1; ++i) {
      const int t = t0 + i - (N - 1);
      if (t >= 0 && t < n_tokens) load_v<V>(h, dtype, (size_t)t * width + c, x[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int t = t0 + i;
    if (t >= n_tokens) return;
    const int s = tok_seq[t], start = seq_start[s], r = t - start;
    if (r < back) {
      if (r == 0)
        convolve_first_rows<T, V>(h, out, width, taps, back + 1, hist + (size_t)slots[s] * hist_stride + c, start, seq_start[s + 1] - start, c);
      continue;
    }
    float acc[V];
    if (N) {
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = x[i + N - 1][e];
#pragma unroll
      for (int j = 0; j < N; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(w[j][e], x[i + j][e], acc[e]);
    } else {
      load_v<V>(h, dtype, (size_t)t * width + c, acc);
      for (int j = 0; j <= back; ++j) {
        float v[V], tw[V];
        load_v<V>(h, dtype, (size_t)(t - back + j) * width + c, v);
        load_v<V>(taps, BN_F32, (size_t)j * width + c, tw);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(tw[e], v[e], acc[e]);
      }
    }
    store_v<V>(out, dtype, (size_t)t * width + c, acc);
  }
}

extern "C" int bn_input_convolution(const void* h, void* out, int dtype, int n_tokens, int width, const float* taps, int n_taps,
                                    void* hist, long long hist_stride, const int* tok_seq, const int* seq_start, const int* slots,
                                    cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  if (!h || !out || h == out || !taps || width <= 0 || n_taps < 1 || n_taps > ST_MAX_TAPS || !tok_seq || !seq_start || !slots ||
      (n_taps > 1 && !hist))
    return BN_ERR_BAD_ARG;
  const bool vec = width % 8 == 0 && hist_stride % 8 == 0 && !(((uintptr_t)h | (uintptr_t)out | (uintptr_t)taps | (uintptr_t)hist) & 15);
#define ST_CONV(TT, VV, NN, RR)                                                                                                  \
  do {                                                                                                                           \
    if ((n_tokens + RR - 1) / RR > 65535) return BN_ERR_BAD_ARG;                                                                 \
    BN_LAUNCH((input_convolution_kernel<TT, VV, NN, RR>), dim3((width / VV + 127) / 128, (n_tokens + RR - 1) / RR), 128, 0, stream, \
              (const TT*)h, (TT*)out, width, n_tokens, taps, n_taps, (TT*)hist, (size_t)hist_stride, tok_seq, seq_start, slots); \
  } while (0)
#define ST_CONV_T(TT)                                   \
  do {                                                  \
    if (!vec) ST_CONV(TT, 1, 0, 4);                     \
    else if (n_taps == 2) ST_CONV(TT, 4, 2, 4);         \
    else if (n_taps == 3) ST_CONV(TT, 4, 3, 4);         \
    else if (n_taps == 4) ST_CONV(TT, 4, 4, 4);         \
    else ST_CONV(TT, 4, 0, 4);                          \
  } while (0)
  if (dtype == BN_F32) ST_CONV_T(float);
  else if (dtype == BN_BF16) ST_CONV_T(__nv_bfloat16);
  else return BN_ERR_BAD_ARG;
#undef ST_CONV_T
#undef ST_CONV
  return BN_OK;
}
