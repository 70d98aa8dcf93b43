// Mixture of experts with sigmoid scores: routing, and the expert products for few tokens.
//
//   z = W_router h (float32), s = sigmoid(z); each token takes the `top` experts with the largest
//   scores; its weight for an expert is that expert's score, taken as it is (or renormalised over the
//   chosen ones), and multiplies either the expert's input or its output.  Optionally the choice goes by
//   the scores plus a correction per expert, and only among the best of several equal groups of experts.
//   Ids from n_real on are identity experts: their output is the token's row h itself.
//
//   bn_moe_route     ids[t][k], weights[t][k] for every token
//   bn_moe_gate_up   y[t * top + k] = act(W_gate[e] x, W_up[e] x) with x = h[t] (times the weight, when it
//                    scales the input) for e = ids[t][k]
//   bn_moe_down      out[t] = sum_k (weight) W_down[e] y[t * top + k] (+ what a shared expert gave), float32
//   bn_moe_scale_rows  x[t * top + k] = weight[t][k] * h[t], for the path that multiplies expert by expert
//
// The two product kernels stream an expert's matrices once per (token, expert) and are meant for the
// few rows of a decode step; they read everything they need from device memory, so a step that
// uses them can be recorded.  With many rows the tokens are sorted by expert instead and every
// expert's rows go through the library's ordinary products (parts/moe.py).
//
// The activation is the clamped gated unit of act.cu: g = min(gate, limit), u = clamp(up, +-limit),
// y = g * sigmoid(slope * g) * (u + 1); or act(gate) * up; or, without a gate matrix, the square of relu(up).
#include "common.cuh"

#define MOE_MAX_EXPERTS 1024

// Shared memory beyond the default 48 KB is asked for once per kernel and size (up to MOE_SMEM_MAX bytes).
#define MOE_SMEM_MAX (200 * 1024)
template <typename K>
static int moe_grant_smem(K kernel, size_t smem, size_t* granted) {
  if (smem > MOE_SMEM_MAX) return BN_ERR_BAD_ARG;
  if (smem > 48 * 1024 && smem > *granted) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return BN_ERR_LAUNCH + (int)e;
    *granted = smem;
  }
  return BN_OK;
}

// How a token's experts are chosen when not by their logits alone: by the scores plus `correction` [n_experts], among the
// experts of the `keep` groups (of `groups` equal ones, neighbours) whose largest such number is largest.
struct MoeChoice {
  const float* correction;  // null: the order of the logits
  int groups, keep;
  float* gate;  // [tokens]: the logistic function of the product with the router's row n_experts, or null
};

// The best of n numbers in shared memory and its place (the lowest among equals; 0 where there is none), by one warp
__device__ __forceinline__ int moe_pick(const float* v, int n, int lane, float* best_out) {
  float best = -INFINITY;
  int arg = n;
  for (int e = lane; e < n; e += 32)
    if (v[e] > best) { best = v[e]; arg = e; }
  for (int o = 16; o > 0; o >>= 1) {
    float ob = __shfl_xor_sync(0xffffffffu, best, o);
    int oa = __shfl_xor_sync(0xffffffffu, arg, o);
    if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
  }
  *best_out = best;
  return arg < n ? arg : 0;
}

// A token's experts from its logits z [n_experts] (which are used up), by one warp; score and group_best: working space of
// n_experts numbers each.
__device__ __forceinline__ void moe_choose(float* z, float* score, float* group_best, int n_experts, int top, int renormalise, int softmax,
                                           float weight_scale, float sum_eps, const MoeChoice& choice, int t, int lane,
                                           int* __restrict__ ids, float* __restrict__ weights) {
  // softmax scores: e^(z - max) over the sum of all experts' (the order of the scores is the logits')
  float z_max = -INFINITY, z_sum = 0.f;
  if (softmax) {
    for (int e = lane; e < n_experts; e += 32) z_max = fmaxf(z_max, z[e]);
    z_max = warp_max(z_max);
    for (int e = lane; e < n_experts; e += 32) z_sum += expf(z[e] - z_max);
    z_sum = warp_sum(z_sum);
  }
  if (choice.correction) {
    // z becomes the choice scores, the scores themselves wait in score
    for (int e = lane; e < n_experts; e += 32) {
      const float s = softmax ? expf(z[e] - z_max) / z_sum : 1.0f / (1.0f + expf(-z[e]));
      score[e] = s;
      z[e] = s + choice.correction[e];
    }
    __syncwarp();
    if (choice.keep < choice.groups) {
      const int size = n_experts / choice.groups;
      for (int g = lane; g < choice.groups; g += 32) {
        float m = -INFINITY;
        for (int e = g * size; e < (g + 1) * size; ++e) m = fmaxf(m, z[e]);
        group_best[g] = m;
      }
      __syncwarp();
      // the groups that stay are marked by +infinity, which is looked past
      for (int k = 0; k < choice.keep; ++k) {
        float best = -INFINITY;
        int arg = choice.groups;
        for (int g = lane; g < choice.groups; g += 32)
          if (group_best[g] > best && group_best[g] != INFINITY) { best = group_best[g]; arg = g; }
        for (int o = 16; o > 0; o >>= 1) {
          float ob = __shfl_xor_sync(0xffffffffu, best, o);
          int oa = __shfl_xor_sync(0xffffffffu, arg, o);
          if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
        }
        if (lane == 0 && arg < choice.groups) group_best[arg] = INFINITY;
        __syncwarp();
      }
      for (int e = lane; e < n_experts; e += 32)
        if (group_best[e / size] != INFINITY) z[e] = -INFINITY;
      __syncwarp();
    }
  }
  float total = 0.f;
  for (int k = 0; k < top; ++k) {
    // the largest logit (or choice score) left; among equal ones the lowest index
    float best;
    const int arg = moe_pick(z, n_experts, lane, &best);
    float s = choice.correction ? score[arg] : softmax ? expf(best - z_max) / z_sum : 1.0f / (1.0f + expf(-best));
    __syncwarp();
    total += s;
    if (lane == 0) {
      ids[(size_t)t * top + k] = arg;
      weights[(size_t)t * top + k] = s;
      z[arg] = -INFINITY;
    }
    __syncwarp();
  }
  __syncwarp();
  if (lane < top && (renormalise || weight_scale != 1.0f)) {
    float wt = weights[(size_t)t * top + lane];
    if (renormalise) wt /= total + sum_eps;
    weights[(size_t)t * top + lane] = wt * weight_scale;
  }
}

template <typename T, typename W>
__global__ void moe_route_kernel(const T* __restrict__ h, int width, const W* __restrict__ w, const float* __restrict__ bias,
                                 int n_experts, int top,
                                 int renormalise, int softmax, float weight_scale, float sum_eps, MoeChoice choice,
                                 int* __restrict__ ids, float* __restrict__ weights) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float z[MOE_MAX_EXPERTS], score[MOE_MAX_EXPERTS], group_best[MOE_MAX_EXPERTS];
  extern __shared__ __align__(16) float xs[];  // width
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  const T* row = h + (size_t)t * width;
  for (int c = threadIdx.x; c < width; c += blockDim.x) xs[c] = to_f32<T>(row[c]);
  __syncthreads();
  for (int e = warp; e < n_experts + (choice.gate ? 1 : 0); e += n_warps) {
    float dot = warp_dot(xs, w + (size_t)e * width, width, lane);
    if (lane == 0) {
      if (e == n_experts) choice.gate[t] = 1.0f / (1.0f + expf(-dot));
      else z[e] = bias ? dot + bias[e] : dot;
    }
  }
  __syncthreads();
  if (warp == 0) {
    moe_choose(z, score, group_best, n_experts, top, renormalise, softmax, weight_scale, sum_eps, choice, t, lane, ids, weights);
  }
}

// The same from logits that a product has left: a warp per token.  logits [tokens, stride] float32; with choice.gate the logit of
// the gate follows the experts'.
#define MOE_CHOOSE_WARPS 4
__global__ void moe_choose_kernel(const float* __restrict__ logits, int stride, int n_tokens, const float* __restrict__ bias, int n_experts,
                                  int top, int renormalise, int softmax, float weight_scale, float sum_eps, MoeChoice choice,
                                  int* __restrict__ ids, float* __restrict__ weights) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];  // per warp: logits, scores, groups
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x * MOE_CHOOSE_WARPS + warp;
  if (t >= n_tokens) return;
  float* z = sm + (size_t)warp * 3 * n_experts;
  const float* row = logits + (size_t)t * stride;
  for (int e = lane; e < n_experts; e += 32) z[e] = bias ? row[e] + bias[e] : row[e];
  if (choice.gate && lane == 0) choice.gate[t] = 1.0f / (1.0f + expf(-row[n_experts]));
  __syncwarp();
  moe_choose(z, z + n_experts, z + 2 * n_experts, n_experts, top, renormalise, softmax, weight_scale, sum_eps, choice, t, lane, ids, weights);
}

extern "C" int bn_moe_choose(const float* logits, int stride, int n_tokens, const float* bias, int n_experts, int top, int renormalise,
                             int softmax, float weight_scale, float sum_eps, const float* correction, int groups, int keep, float* gate,
                             int* ids, float* weights, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  if (!logits || !ids || !weights || n_experts <= 0 || n_experts > MOE_MAX_EXPERTS || stride < n_experts + (gate ? 1 : 0) || top <= 0 ||
      top > n_experts || top > 32 || groups <= 0 || n_experts % groups || keep <= 0 || keep > groups || (keep < groups && !correction))
    return BN_ERR_BAD_ARG;
  const MoeChoice choice = {correction, groups, keep, gate};
  const size_t smem = (size_t)MOE_CHOOSE_WARPS * 3 * n_experts * sizeof(float);  // at most 48 KB
  BN_LAUNCH(moe_choose_kernel, (n_tokens + MOE_CHOOSE_WARPS - 1) / MOE_CHOOSE_WARPS, MOE_CHOOSE_WARPS * 32, smem, stream, logits, stride, n_tokens,
            bias, n_experts, top, renormalise, softmax, weight_scale, sum_eps, choice, ids, weights);
  return BN_OK;
}

// softmax: the scores are the softmax over all experts instead of each logit's logistic function; the chosen
// experts' scores are divided by their sum + sum_eps with `renormalise`, then multiplied by weight_scale.  bias
// [n_experts] float32 (or null) is added to the logits before anything is chosen.  correction [n_experts] float32 (or null):
// the choice goes by score + correction, and with keep < groups only among the experts of the best `keep` of `groups` equal
// groups of neighbours (a group counts by its best).  gate [n_tokens] (or null): w then has a row n_experts, and gate
// receives the logistic function of its product with h.
extern "C" int bn_moe_route_ex(const void* h, int h_dtype, int n_tokens, int width, const void* w, int w_dtype, const float* bias,
                               int n_experts, int top, int renormalise, int softmax, float weight_scale, float sum_eps,
                               const float* correction, int groups, int keep, float* gate, int* ids, float* weights,
                               cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  if (!h || !w || !ids || !weights || width <= 0 || n_experts <= 0 || n_experts > MOE_MAX_EXPERTS || top <= 0 ||
      top > n_experts || top > 32 ||
      groups <= 0 || n_experts % groups || keep <= 0 || keep > groups || (keep < groups && !correction))
    return BN_ERR_BAD_ARG;
  const MoeChoice choice = {correction, groups, keep, gate};
  const size_t smem = (size_t)width * sizeof(float);
  static size_t granted[3] = {0, 0, 0};
  const size_t beside = 3 * MOE_MAX_EXPERTS * sizeof(float);  // the kernel's static part counts towards the default too
  if (smem + beside > 48 * 1024) {
    const int rc = h_dtype == BN_F32 ? moe_grant_smem(moe_route_kernel<float, float>, smem + beside, &granted[0])
                   : w_dtype == BN_F32 ? moe_grant_smem(moe_route_kernel<__nv_bfloat16, float>, smem + beside, &granted[1])
                                       : moe_grant_smem(moe_route_kernel<__nv_bfloat16, __nv_bfloat16>, smem + beside, &granted[2]);
    if (rc != BN_OK) return rc;
  }
  if (h_dtype == BN_F32 && w_dtype == BN_F32)
    BN_LAUNCH((moe_route_kernel<float, float>), n_tokens, 256, smem, stream, (const float*)h, width, (const float*)w, bias,
              n_experts, top, renormalise, softmax, weight_scale, sum_eps, choice, ids, weights);
  else if (h_dtype == BN_BF16 && w_dtype == BN_BF16)
    BN_LAUNCH((moe_route_kernel<__nv_bfloat16, __nv_bfloat16>), n_tokens, 256, smem, stream, (const __nv_bfloat16*)h, width,
              (const __nv_bfloat16*)w, bias, n_experts, top, renormalise, softmax, weight_scale, sum_eps, choice, ids, weights);
  else if (h_dtype == BN_BF16 && w_dtype == BN_F32)
    BN_LAUNCH((moe_route_kernel<__nv_bfloat16, float>), n_tokens, 256, smem, stream, (const __nv_bfloat16*)h, width,
              (const float*)w, bias, n_experts, top, renormalise, softmax, weight_scale, sum_eps, choice, ids, weights);
  else
    return BN_ERR_BAD_ARG;
  BN_CHECK_LAUNCH();
  return BN_OK;
}

extern "C" int bn_moe_route(const void* h, int h_dtype, int n_tokens, int width, const void* w, int w_dtype,
                            int n_experts, int top, int renormalise, int* ids, float* weights, cudaStream_t stream) {
  return bn_moe_route_ex(h, h_dtype, n_tokens, width, w, w_dtype, nullptr, n_experts, top, renormalise, 0, 1.0f, 0.0f, nullptr, 1, 1, nullptr,
                         ids, weights, stream);
}

#define MOE_THREADS 256
#define MOE_ROWS_PER_BLOCK 32  // outputs per block of the product kernels

// grid (tokens * top, ceil(ff / MOE_ROWS_PER_BLOCK)); row j of expert e's gate matrix lies at
// w_gate + e * expert_stride + j * width, of its up matrix at w_up + the same (so that one tensor
// [experts, 2 * ff, width] with the gate rows first serves both)
template <typename T>
__global__ void moe_gate_up_kernel(const T* __restrict__ h, int width, const int* __restrict__ ids,
                                   const float* __restrict__ weights, int scale_input, const T* __restrict__ w_gate,
                                   const T* __restrict__ w_up, size_t expert_stride, int ff, int top, float limit,
                                   float slope, int act, int n_real, T* __restrict__ y) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float xs[];  // width
  const int item = blockIdx.x, t = item / top;
  const int e = ids[item];
  if (e >= n_real) return;  // an identity expert
  const float wt = scale_input ? weights[item] : 1.0f;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  // the expert's input in the compute type, as the path that sorts tokens by expert stores it
  for (int c = threadIdx.x; c < width; c += blockDim.x)
    xs[c] = to_f32<T>(from_f32<T>(to_f32<T>(h[(size_t)t * width + c]) * wt));
  __syncthreads();
  const int j0 = blockIdx.y * MOE_ROWS_PER_BLOCK, j1 = min(ff, j0 + MOE_ROWS_PER_BLOCK);
  // a warp takes four neighbouring rows of both matrices at a time
  for (int j = j0 + warp * 4; j < j1; j += n_warps * 4) {
    float g4[4] = {0.f, 0.f, 0.f, 0.f}, u4[4];
    const T* gr = w_gate ? w_gate + (size_t)e * expert_stride + (size_t)j * width : nullptr;
    const T* ur = w_up + (size_t)e * expert_stride + (size_t)j * width;
    if (j + 4 <= j1) {
      if (gr) warp_dot_rows<4>(xs, gr, (size_t)width, width, lane, g4);
      warp_dot_rows<4>(xs, ur, (size_t)width, width, lane, u4);
    } else {
      for (int r = 0; r < j1 - j; ++r) {
        if (gr) g4[r] = warp_dot(xs, gr + (size_t)r * width, width, lane);
        u4[r] = warp_dot(xs, ur + (size_t)r * width, width, lane);
      }
    }
    if (lane < 4 && j + lane < j1) {
      // the products' results pass through the compute type, as they do on the sorted path
      float g = lane == 0 ? g4[0] : lane == 1 ? g4[1] : lane == 2 ? g4[2] : g4[3];
      float u = lane == 0 ? u4[0] : lane == 1 ? u4[1] : lane == 2 ? u4[2] : u4[3];
      g = to_f32<T>(from_f32<T>(g));
      u = to_f32<T>(from_f32<T>(u));
      if (!w_gate) {  // the unit without a gate
        y[(size_t)item * ff + j + lane] = from_f32<T>(relu_squared(u));
      } else if (act >= 0) {  // the plain gated unit: act(g) * u
        y[(size_t)item * ff + j + lane] = from_f32<T>(glu_activation(g, act) * u);
      } else {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        y[(size_t)item * ff + j + lane] = from_f32<T>(g / (1.0f + expf(-slope * g)) * (u + 1.0f));
      }
    }
  }
}

// grid (tokens, ceil(width / MOE_ROWS_PER_BLOCK)); w_down: [experts, width, ff]
template <typename T>
__global__ void moe_down_kernel(const T* __restrict__ y, int ff, const int* __restrict__ ids,
                                const float* __restrict__ weights, int scale_output, const T* __restrict__ w_down,
                                int width, int top, const void* __restrict__ add, int add_dtype,
                                const float* __restrict__ add_scale, int n_real, const T* __restrict__ h, float* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float ys[];  // top * ff: the token's activations, expert by expert
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  for (int k = 0; k < top; ++k) {
    if (ids[(size_t)t * top + k] >= n_real) continue;  // an identity expert has no activations
    const size_t at = ((size_t)t * top + k) * ff;
    for (int i = threadIdx.x; i < ff; i += blockDim.x) ys[(size_t)k * ff + i] = to_f32<T>(y[at + i]);
  }
  __syncthreads();
  const int c0 = blockIdx.y * MOE_ROWS_PER_BLOCK, c1 = min(width, c0 + MOE_ROWS_PER_BLOCK);
  for (int c = c0 + warp * 4; c < c1; c += n_warps * 4) {
    float total[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k = 0; k < top; ++k) {
      const int e = ids[(size_t)t * top + k];
      const T* wr = w_down + ((size_t)e * width + c) * ff;
      float d4[4] = {0.f, 0.f, 0.f, 0.f};
      if (e >= n_real) {
        for (int r = 0; r < min(4, c1 - c); ++r) d4[r] = to_f32<T>(h[(size_t)t * width + c + r]);
      } else if (c + 4 <= c1) {
        warp_dot_rows<4>(ys + (size_t)k * ff, wr, (size_t)ff, ff, lane, d4);
      } else {
        for (int r = 0; r < c1 - c; ++r) d4[r] = warp_dot(ys + (size_t)k * ff, wr + (size_t)r * ff, ff, lane);
      }
      const float wt = scale_output ? weights[(size_t)t * top + k] : 1.0f;
#pragma unroll
      for (int r = 0; r < 4; ++r) total[r] += d4[r] * wt;
    }
    if (lane < 4 && c + lane < c1) {
      float v = lane == 0 ? total[0] : lane == 1 ? total[1] : lane == 2 ? total[2] : total[3];
      if (add) v += load_as_f32(add, add_dtype, (size_t)t * width + c + lane) * (add_scale ? add_scale[t] : 1.0f);
      out[(size_t)t * width + c + lane] = v;
    }
  }
}

// act < 0: the clamped unit with `limit` and `slope`; act >= 0 (BN_ACT_*): act(gate) * up without clamps; w_gate null: the
// square of relu(up).  Ids from n_real on are identity experts, which have nothing to do here.
extern "C" int bn_moe_gate_up_ex(const void* h, int dtype, int n_tokens, int width, const int* ids, const float* weights,
                                 int scale_input, const void* w_gate, const void* w_up, long long expert_stride, int ff, int top,
                                 float limit, float slope, int act, int n_real, void* y, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  if (!h || !ids || !weights || !w_up || !y || width <= 0 || ff <= 0 || top <= 0) return BN_ERR_BAD_ARG;
  size_t smem = (size_t)width * sizeof(float);
  static size_t granted[2] = {0, 0};
  int rc = dtype == BN_F32 ? moe_grant_smem(moe_gate_up_kernel<float>, smem, &granted[0])
                           : moe_grant_smem(moe_gate_up_kernel<__nv_bfloat16>, smem, &granted[1]);
  if (rc != BN_OK) return rc;
  dim3 grid(n_tokens * top, (ff + MOE_ROWS_PER_BLOCK - 1) / MOE_ROWS_PER_BLOCK);
  if (dtype == BN_F32)
    BN_LAUNCH(moe_gate_up_kernel<float>, grid, MOE_THREADS, smem, stream, (const float*)h, width, ids, weights, scale_input,
              (const float*)w_gate, (const float*)w_up, (size_t)expert_stride, ff, top, limit, slope, act, n_real, (float*)y);
  else if (dtype == BN_BF16)
    BN_LAUNCH(moe_gate_up_kernel<__nv_bfloat16>, grid, MOE_THREADS, smem, stream, (const __nv_bfloat16*)h, width, ids,
              weights, scale_input, (const __nv_bfloat16*)w_gate, (const __nv_bfloat16*)w_up, (size_t)expert_stride, ff, top, limit,
              slope, act, n_real, (__nv_bfloat16*)y);
  else
    return BN_ERR_BAD_ARG;
  BN_CHECK_LAUNCH();
  return BN_OK;
}

extern "C" int bn_moe_gate_up(const void* h, int dtype, int n_tokens, int width, const int* ids, const float* weights,
                              int scale_input, const void* w_gate, const void* w_up, long long expert_stride, int ff, int top,
                              float limit, float slope, void* y, cudaStream_t stream) {
  return bn_moe_gate_up_ex(h, dtype, n_tokens, width, ids, weights, scale_input, w_gate, w_up, expert_stride, ff, top, limit, slope,
                           -1, 1 << 30, y, stream);
}

// add_scale [n_tokens] (or null): a factor on the token's row of `add`; ids from n_real on are identity experts, whose output is
// the token's row of h [n_tokens, width]
extern "C" int bn_moe_down(const void* y, int dtype, int n_tokens, int ff, const int* ids, const float* weights,
                           int scale_output, const void* w_down, int width, int top, const void* add, int add_dtype,
                           const float* add_scale, int n_real, const void* h, float* out, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  if (!y || !ids || !weights || !w_down || !out || width <= 0 || ff <= 0 || top <= 0) return BN_ERR_BAD_ARG;
  dim3 grid(n_tokens, (width + MOE_ROWS_PER_BLOCK - 1) / MOE_ROWS_PER_BLOCK);
  const size_t smem = (size_t)top * ff * sizeof(float);
  static size_t granted[2] = {0, 0};
  int rc = dtype == BN_F32 ? moe_grant_smem(moe_down_kernel<float>, smem, &granted[0])
                           : moe_grant_smem(moe_down_kernel<__nv_bfloat16>, smem, &granted[1]);
  if (rc != BN_OK) return rc;
  if (dtype == BN_F32)
    BN_LAUNCH(moe_down_kernel<float>, grid, MOE_THREADS, smem, stream, (const float*)y, ff, ids, weights, scale_output,
              (const float*)w_down, width, top, add, add_dtype, add_scale, n_real, (const float*)h, out);
  else if (dtype == BN_BF16)
    BN_LAUNCH(moe_down_kernel<__nv_bfloat16>, grid, MOE_THREADS, smem, stream, (const __nv_bfloat16*)y, ff, ids, weights,
              scale_output, (const __nv_bfloat16*)w_down, width, top, add, add_dtype, add_scale, n_real, (const __nv_bfloat16*)h, out);
  else
    return BN_ERR_BAD_ARG;
  BN_CHECK_LAUNCH();
  return BN_OK;
}

// ---- sorting tokens by expert (many rows) --------------------------------------------------------
// counts[e] = how many (token, k) items chose expert e; one thread per item.  Identity experts (from n_real on) are not sorted.
__global__ void moe_count_kernel(const int* __restrict__ ids, int n_items, int n_real, int* __restrict__ counts) {
  pdl_launch_dependents();
  pdl_wait();
  int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n_items && ids[i] < n_real) atomicAdd(&counts[ids[i]], 1);
}

// offsets[e] = first row of expert e in the sorted order: the experts' rows packed one behind another
// (cap == 0; offsets[n_experts] = n_items), or every expert in a block of cap rows of its own; one block.
__global__ void moe_offsets_kernel(const int* __restrict__ counts, int n_experts, int cap, int* __restrict__ offsets,
                                   int* __restrict__ cursor) {
  pdl_launch_dependents();
  pdl_wait();
  if (threadIdx.x == 0) {
    int at = 0;
    for (int e = 0; e < n_experts; ++e) {
      offsets[e] = at;
      cursor[e] = at;
      at += cap > 0 ? cap : counts[e];
    }
    offsets[n_experts] = at;
  }
}

// The same, packed, from the items themselves (counted in shared memory); one block of 1,024 threads.
__global__ void __launch_bounds__(1024) moe_count_offsets_kernel(const int* __restrict__ ids, int n_items, int n_experts,
                                                                 int* __restrict__ offsets, int* __restrict__ cursor) {
  pdl_launch_dependents();
  __shared__ int counts[MOE_MAX_EXPERTS], warp_total[32];
  const int e = threadIdx.x, lane = e & 31, warp = e >> 5;
  counts[e] = 0;
  __syncthreads();
  pdl_wait();
  for (int i = e; i < n_items; i += 1024) {
    const int id = ids[i];
    if (id < n_experts) atomicAdd(&counts[id], 1);
  }
  __syncthreads();
  const int mine = counts[e];
  int upto = mine;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int up = __shfl_up_sync(0xffffffffu, upto, o);
    if (lane >= o) upto += up;
  }
  if (lane == 31) warp_total[warp] = upto;
  __syncthreads();
  for (int w = 0; w < warp; ++w) upto += warp_total[w];
  if (e < n_experts) {
    offsets[e] = cursor[e] = upto - mine;
    if (e == n_experts - 1) offsets[n_experts] = upto;
  }
}

// place[i] = row of item i in the sorted order, and x_sorted[place[i]] = weight * h[token of i] (or h itself).
// Rows of one expert come in any order; every row is computed alone, so the order changes no result.
template <typename T>
__global__ void moe_scatter_kernel(const T* __restrict__ h, int width, const int* __restrict__ ids,
                                   const float* __restrict__ weights, int scale_input, int top, int n_real, int* __restrict__ cursor,
                                   int* __restrict__ place, T* __restrict__ x_sorted) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ int row;
  const int item = blockIdx.x, t = item / top;
  if (ids[item] >= n_real) {  // an identity expert: no row
    if (threadIdx.x == 0) place[item] = -1;
    return;
  }
  if (threadIdx.x == 0) {
    row = atomicAdd(&cursor[ids[item]], 1);
    place[item] = row;
  }
  __syncthreads();
  const float wt = scale_input ? weights[item] : 1.0f;
  constexpr int V = 16 / (int)sizeof(T);
  const T* src = h + (size_t)t * width;
  T* dst = x_sorted + (size_t)row * width;
  if (width % V == 0 && (((uintptr_t)h | (uintptr_t)x_sorted) & 15) == 0) {  // rows of whole 16-byte pieces
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
      uint4 raw = *reinterpret_cast<const uint4*>(src + c);
      if (scale_input) {
        T* v = reinterpret_cast<T*>(&raw);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = from_f32<T>(to_f32<T>(v[e]) * wt);
      }
      *reinterpret_cast<uint4*>(dst + c) = raw;
    }
    return;
  }
  for (int c = threadIdx.x; c < width; c += blockDim.x) dst[c] = from_f32<T>(to_f32<T>(src[c]) * wt);
}

// out[t] = sum_k (weight) y_sorted[place[t * top + k]] (+ add_scale[t] add[t]), float32; a place below zero: the row of h
template <typename T>
__global__ void moe_gather_kernel(const T* __restrict__ y_sorted, int width, const int* __restrict__ place,
                                  const float* __restrict__ weights, int scale_output, int top,
                                  const void* __restrict__ add, int add_dtype, const float* __restrict__ add_scale,
                                  const T* __restrict__ h, float* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  constexpr int V = 16 / (int)sizeof(T);
  if (width % V == 0 && (!add || add_dtype == BN_F32) &&
      (((uintptr_t)y_sorted | (uintptr_t)h | (uintptr_t)out | (uintptr_t)add) & 15) == 0) {  // rows of whole 16-byte pieces
    const float factor = add_scale ? add_scale[t] : 1.0f;
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
      float total[V];
#pragma unroll
      for (int e = 0; e < V; ++e) total[e] = 0.f;
      for (int k = 0; k < top; ++k) {
        const int row = place[(size_t)t * top + k];
        const float wt = scale_output ? weights[(size_t)t * top + k] : 1.0f;
        const T* src = row >= 0 ? y_sorted + (size_t)row * width : h ? h + (size_t)t * width : nullptr;
        if (!src) continue;
        const uint4 raw = *reinterpret_cast<const uint4*>(src + c);
        const T* v = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int e = 0; e < V; ++e) total[e] = scale_output ? fmaf(to_f32<T>(v[e]), wt, total[e]) : total[e] + to_f32<T>(v[e]);
      }
      float4* dst = reinterpret_cast<float4*>(out + (size_t)t * width + c);
#pragma unroll
      for (int e = 0; e < V; e += 4) {
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        if (add) a = *reinterpret_cast<const float4*>((const float*)add + (size_t)t * width + c + e);
        dst[e / 4] = make_float4(fmaf(a.x, factor, total[e]), fmaf(a.y, factor, total[e + 1]), fmaf(a.z, factor, total[e + 2]),
                                 fmaf(a.w, factor, total[e + 3]));
      }
    }
    return;
  }
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
      const int row = place[(size_t)t * top + k];
      float v = row >= 0 ? to_f32<T>(y_sorted[(size_t)row * width + c]) : h ? to_f32<T>(h[(size_t)t * width + c]) : 0.f;
      total += scale_output ? v * weights[(size_t)t * top + k] : v;
    }
    if (add) total += load_as_f32(add, add_dtype, (size_t)t * width + c) * (add_scale ? add_scale[t] : 1.0f);
    out[(size_t)t * width + c] = total;
  }
}

// counts: [n_experts], zeroed by the caller: how many (token, expert) items chose each expert (ids from n_experts on are
// identity experts and not counted)
extern "C" int bn_moe_count(const int* ids, int n_items, int n_experts, int* counts, cudaStream_t stream) {
  if (n_items <= 0) return BN_OK;
  if (!ids || !counts) return BN_ERR_BAD_ARG;
  BN_LAUNCH(moe_count_kernel, (n_items + 255) / 256, 256, 0, stream, ids, n_items, n_experts, counts);
  BN_CHECK_LAUNCH();
  return BN_OK;
}

// counts as bn_moe_count left them (or null: counted here; cap == 0 then); offsets: [n_experts + 1]; cursor: [n_experts]; place: [n_items];
// x_sorted: [n_items, width] (cap == 0) or [n_experts * cap, width] (cap >= the largest count)
extern "C" int bn_moe_scatter(const void* h, int dtype, int n_tokens, int width, const int* ids, const float* weights,
                              int scale_input, int top, int n_experts, int cap, const int* counts, int* offsets,
                              int* cursor, int* place, void* x_sorted, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  if (!h || !ids || !weights || (!counts && (cap > 0 || n_experts > MOE_MAX_EXPERTS)) || !offsets || !cursor || !place || !x_sorted || width <= 0 || top <= 0 ||
      n_experts <= 0 || cap < 0)
    return BN_ERR_BAD_ARG;
  int n_items = n_tokens * top;
  if (counts)
    BN_LAUNCH(moe_offsets_kernel, 1, 32, 0, stream, counts, n_experts, cap, offsets, cursor);
  else
    BN_LAUNCH(moe_count_offsets_kernel, 1, 1024, 0, stream, ids, n_items, n_experts, offsets, cursor);
  if (dtype == BN_F32)
    BN_LAUNCH(moe_scatter_kernel<float>, n_items, 128, 0, stream, (const float*)h, width, ids, weights, scale_input, top, n_experts,
              cursor, place, (float*)x_sorted);
  else if (dtype == BN_BF16)
    BN_LAUNCH(moe_scatter_kernel<__nv_bfloat16>, n_items, 128, 0, stream, (const __nv_bfloat16*)h, width, ids, weights,
              scale_input, top, n_experts, cursor, place, (__nv_bfloat16*)x_sorted);
  else
    return BN_ERR_BAD_ARG;
  BN_CHECK_LAUNCH();
  return BN_OK;
}

extern "C" int bn_moe_gather(const void* y_sorted, int dtype, int n_tokens, int width, const int* place,
                             const float* weights, int scale_output, int top, const void* add, int add_dtype,
                             const float* add_scale, const void* h, float* out, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  if (!y_sorted || !place || !weights || !out || width <= 0 || top <= 0) return BN_ERR_BAD_ARG;
  if (dtype == BN_F32)
    BN_LAUNCH(moe_gather_kernel<float>, n_tokens, 256, 0, stream, (const float*)y_sorted, width, place, weights,
              scale_output, top, add, add_dtype, add_scale, (const float*)h, out);
  else if (dtype == BN_BF16)
    BN_LAUNCH(moe_gather_kernel<__nv_bfloat16>, n_tokens, 256, 0, stream, (const __nv_bfloat16*)y_sorted, width, place,
              weights, scale_output, top, add, add_dtype, add_scale, (const __nv_bfloat16*)h, out);
  else
    return BN_ERR_BAD_ARG;
  BN_CHECK_LAUNCH();
  return BN_OK;
}

// Experts by a table instead of a router: token id -> the `top` experts of its row, each with the same weight.
// table [vocab, table_stride] int32; an id outside the table, or an entry outside the experts, takes expert 0
// with weight 0 (it adds nothing).
__global__ void moe_table_route_kernel(const int* __restrict__ tokens, int n_tokens, const int* __restrict__ table, int vocab,
                                       int table_stride, int top, int n_experts, float weight, int* __restrict__ ids,
                                       float* __restrict__ weights) {
  pdl_launch_dependents();
  pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n_tokens * top) return;
  const int t = i / top, k = i - t * top;
  const int tok = tokens[t];
  int e = tok >= 0 && tok < vocab ? table[(size_t)tok * table_stride + k] : -1;
  const bool ok = e >= 0 && e < n_experts;
  ids[i] = ok ? e : 0;
  weights[i] = ok ? weight : 0.f;
}

extern "C" int bn_moe_table_route(const int* tokens, int n_tokens, const int* table, int vocab, int table_stride, int top,
                                  int n_experts, float weight, int* ids, float* weights, cudaStream_t stream) {
  if (n_tokens <= 0) return BN_OK;
  if (!tokens || !table || !ids || !weights || top <= 0 || top > table_stride || vocab <= 0 || n_experts <= 0) return BN_ERR_BAD_ARG;
  BN_LAUNCH(moe_table_route_kernel, (n_tokens * top + 255) / 256, 256, 0, stream, tokens, n_tokens, table, vocab, table_stride, top,
            n_experts, weight, ids, weights);
  BN_CHECK_LAUNCH();
  return BN_OK;
}
