// Keys and values per head from cached latents, for runs of new tokens (bfloat16): the rows [latent | rotated key part] that a
// step's tokens see are read back from the pages, two products make every head's unrotated keys and values of the latents,
// and these go, with the shared rotated part behind each head's keys, into scratch pages that the attention kernels for runs
// of tokens read as if they were the cache.
//
//   bn_latent_gather  the latents of the seen positions, side by side: [seen, rank]
//   bn_latent_pages   keys [pages, heads, 64, dim + rot], values [pages, heads, 64, vdim]
#include "common.cuh"

// The cache row of seen position i
__device__ __forceinline__ const __nv_bfloat16* latent_row(const __nv_bfloat16* cache, int row, const int* seen_seq, const int* seen_pos,
                                                           const int* slots, const int* page_table, int pt_stride, int i) {
  const int p = seen_pos[i];
  return cache + ((size_t)page_table[(size_t)slots[seen_seq[i]] * pt_stride + p / BN_PAGE] * BN_PAGE + p % BN_PAGE) * row;
}

__global__ void latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, int row, int rank, const int* __restrict__ seen_seq,
                                     const int* __restrict__ seen_pos, int n_seen, const int* __restrict__ slots,
                                     const int* __restrict__ page_table, int pt_stride, __nv_bfloat16* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int i = blockIdx.x * blockDim.y + threadIdx.y;
  if (i >= n_seen) return;
  const __nv_bfloat16* src = latent_row(cache, row, seen_seq, seen_pos, slots, page_table, pt_stride, i);
  for (int c = threadIdx.x * 8; c < rank; c += blockDim.x * 8)
    *reinterpret_cast<uint4*>(out + (size_t)i * rank + c) = *reinterpret_cast<const uint4*>(src + c);
}

// A block per seen position; scratch_table [sequences, scratch_stride]: the scratch page of each page of a sequence.
__global__ void latent_pages_kernel(const __nv_bfloat16* __restrict__ keys, const __nv_bfloat16* __restrict__ values,
                                    const __nv_bfloat16* __restrict__ cache, int row, int rank, int heads, int dim, int rot, int vdim,
                                    const int* __restrict__ seen_seq, const int* __restrict__ seen_pos, const int* __restrict__ slots,
                                    const int* __restrict__ page_table, int pt_stride, const int* __restrict__ scratch_table,
                                    int scratch_stride, __nv_bfloat16* __restrict__ k_pages, __nv_bfloat16* __restrict__ v_pages) {
  pdl_launch_dependents();
  pdl_wait();
  const int i = blockIdx.x, pos = seen_pos[i];
  const __nv_bfloat16* turned = latent_row(cache, row, seen_seq, seen_pos, slots, page_table, pt_stride, i) + rank;
  const size_t page = scratch_table[(size_t)seen_seq[i] * scratch_stride + pos / BN_PAGE];
  const int r = pos % BN_PAGE, kd = dim + rot, per_key = kd / 8, per_value = vdim / 8;
  for (int j = threadIdx.x; j < heads * per_key; j += blockDim.x) {
    const int h = j / per_key, c = (j - h * per_key) * 8;
    const __nv_bfloat16* src = c < dim ? keys + ((size_t)i * heads + h) * dim + c : turned + c - dim;
    *reinterpret_cast<uint4*>(k_pages + ((page * heads + h) * BN_PAGE + r) * kd + c) = *reinterpret_cast<const uint4*>(src);
  }
  for (int j = threadIdx.x; j < heads * per_value; j += blockDim.x) {
    const int h = j / per_value, c = (j - h * per_value) * 8;
    *reinterpret_cast<uint4*>(v_pages + ((page * heads + h) * BN_PAGE + r) * vdim + c) =
        *reinterpret_cast<const uint4*>(values + ((size_t)i * heads + h) * vdim + c);
  }
}

// cache: pages of 64 rows of `row` bfloat16 numbers (one key head); seen_seq / seen_pos [n_seen]; out [n_seen, rank].  row and rank
// multiples of 8, 16-byte aligned.
extern "C" int bn_latent_gather(const void* cache, int row, int rank, const int* seen_seq, const int* seen_pos, int n_seen, const int* slots,
                                const int* page_table, int pt_stride, void* out, cudaStream_t stream) {
  if (n_seen <= 0) return BN_OK;
  if (!cache || !seen_seq || !seen_pos || !slots || !page_table || !out || rank <= 0 || rank > row || row % 8 || rank % 8 ||
      (((uintptr_t)cache | (uintptr_t)out) & 15))
    return BN_ERR_BAD_ARG;
  BN_LAUNCH(latent_gather_kernel, (n_seen + 3) / 4, dim3(64, 4), 0, stream, (const __nv_bfloat16*)cache, row, rank, seen_seq, seen_pos, n_seen,
            slots, page_table, pt_stride, (__nv_bfloat16*)out);
  return BN_OK;
}

// keys [n_seen, heads, dim], values [n_seen, heads, vdim]; k_pages [pages, heads, 64, row - rank + dim], v_pages [pages, heads, 64,
// vdim]; rows that no seen position fills are left alone.  All widths multiples of 8, all buffers 16-byte aligned.
extern "C" int bn_latent_pages(const void* keys, const void* values, const void* cache, int row, int rank, int heads, int dim, int vdim,
                               const int* seen_seq, const int* seen_pos, int n_seen, const int* slots, const int* page_table, int pt_stride,
                               const int* scratch_table, int scratch_stride, void* k_pages, void* v_pages, cudaStream_t stream) {
  if (n_seen <= 0) return BN_OK;
  if (!keys || !values || !cache || !seen_seq || !seen_pos || !slots || !page_table || !scratch_table || !k_pages || !v_pages || heads <= 0 ||
      dim <= 0 || vdim <= 0 || rank <= 0 || rank > row || row % 8 || rank % 8 || dim % 8 || vdim % 8 ||
      (((uintptr_t)keys | (uintptr_t)values | (uintptr_t)cache | (uintptr_t)k_pages | (uintptr_t)v_pages) & 15))
    return BN_ERR_BAD_ARG;
  BN_LAUNCH(latent_pages_kernel, n_seen, 256, 0, stream, (const __nv_bfloat16*)keys, (const __nv_bfloat16*)values, (const __nv_bfloat16*)cache, row,
            rank, heads, dim, row - rank, vdim, seen_seq, seen_pos, slots, page_table, pt_stride, scratch_table, scratch_stride,
            (__nv_bfloat16*)k_pages, (__nv_bfloat16*)v_pages);
  return BN_OK;
}
