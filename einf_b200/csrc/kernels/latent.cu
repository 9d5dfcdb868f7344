// Pointwise steps of latent attention: keys and values of a token are one normed latent vector
// c [kv_rank] plus one rotated key part r [rot_dim] shared by all heads; the page cache holds the
// row [c | r] once per token (one key/value "head" of size kv_rank + rot_dim whose first kv_rank
// elements are also the value).  Queries come through a normed latent of their own.
//
//   einf_latent_down_store   from the product [q latent | kv latent | key part] of a token:
//                            RMS norm (weight, eps inside the root) of the query latent -> q_latent_out,
//                            RMS norm of the kv latent and rotation of the key part -> cache row
//   einf_latent_q_store      from the up-projected queries [H, dim + rot_dim]: the unrotated part
//                            -> q_plain [T, H, dim] (it still has to pass the key up-projection),
//                            the rotated part -> q_full [T, H, kv_rank + rot_dim] behind the place
//                            of the absorbed part
//   einf_latent_qkv_store    both at once for queries without a latent of their own, from the one product
//                            [kv latent | key part | queries | a gate logit per head] of a token: the
//                            cache row, the queries' two parts, and sigmoid(gate logit)
//
// Rotation of a pair (u, v) at position p: (u cos a - v sin a, v cos a + u sin a), a = p * inv_freq[i];
// pair i is (i, i + rot_dim / 2), or (2i, 2i + 1) with `interleaved`; cosine and sine carry the factor
// `amplitude`.  A cache row and a query may be longer than kv_rank + rot_dim (einf_latent_qkv_store's `row`): the
// rest is zero, so that a kernel that wants rows of its own size sees the same scores.  Norms, angles and sums are
// 32-bit; values are rounded once, into the output type.  Inputs may be float32 split-K partial sums.
#include "common.cuh"

namespace einf {

// Sum of the partial sums of one element, added in order; the loads go out eight at a time (a consumer
// of a product that was cut sixteen ways would otherwise pay sixteen round trips one after the other).
template <typename TIn>
__device__ __forceinline__ float sum_parts(const TIn* __restrict__ p, int splits, size_t split_stride) {
  float v = 0.f;
  int s = 0;
  for (; s + 8 <= splits; s += 8) {
    float t[8];
#pragma unroll
    for (int u = 0; u < 8; ++u) t[u] = to_float(p[(size_t)(s + u) * split_stride]);
#pragma unroll
    for (int u = 0; u < 8; ++u) v += t[u];
  }
  if (s < splits) {
    float t[8];
#pragma unroll
    for (int u = 0; u < 8; ++u) t[u] = s + u < splits ? to_float(p[(size_t)(s + u) * split_stride]) : 0.f;
#pragma unroll
    for (int u = 0; u < 8; ++u) v += t[u];
  }
  return v;
}

__device__ __forceinline__ void pair_of(int i, int half, int interleaved, int* first, int* second) {
  if (interleaved) {
    *first = 2 * i;
    *second = 2 * i + 1;
  } else {
    *first = i;
    *second = i + half;
  }
}

template <typename TIn, typename T>
__global__ void __launch_bounds__(256)
latent_down_store_kernel(const TIn* __restrict__ down, int splits, size_t split_stride, int q_rank, int kv_rank,
                         int rot_dim, const float* __restrict__ q_norm_weight,
                         const float* __restrict__ kv_norm_weight, float eps, const int* __restrict__ positions,
                         const float* __restrict__ inv_freq, float amplitude, int interleaved,
                         const int* __restrict__ slots, T* __restrict__ q_latent_out, T* __restrict__ cache, int page_size, int num_pages,
                         int* status) {
  extern __shared__ float row[];   // [q_rank + kv_rank + rot_dim]
  __shared__ float scratch[33];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int width = q_rank + kv_rank + rot_dim;
  const TIn* src = down + (size_t)t * width;
  float ss_q = 0.f, ss_kv = 0.f;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float v = sum_parts(src + i, splits, split_stride);
    row[i] = v;
    if (i < q_rank) ss_q += v * v;
    else if (i < q_rank + kv_rank) ss_kv += v * v;
  }
  if (q_rank > 0) {
    const float factor = rsqrtf(block_sum(ss_q, scratch) / (float)q_rank + eps);
    for (int i = threadIdx.x; i < q_rank; i += blockDim.x)
      q_latent_out[(size_t)t * q_rank + i] = from_float<T>(row[i] * factor * q_norm_weight[i]);
  }
  const float factor = rsqrtf(block_sum(ss_kv, scratch) / (float)kv_rank + eps);   // has barriers: row[] is complete
  const int slot = slots ? slots[t] : -1;
  if (slot < 0) return;
  const int page = slot / page_size, offset = slot - page * page_size;
  if (page >= num_pages) {
    if (threadIdx.x == 0) atomicOr(status, kStatusBadPage);
    return;
  }
  T* dst = cache + ((size_t)page * page_size + offset) * (kv_rank + rot_dim);
  const float* latent = row + q_rank;
  for (int i = threadIdx.x; i < kv_rank; i += blockDim.x)
    dst[i] = from_float<T>(latent[i] * factor * kv_norm_weight[i]);
  const float* part = latent + kv_rank;
  const int half = rot_dim >> 1;
  const float pos = (float)positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    int a, b;
    pair_of(i, half, interleaved, &a, &b);
    float sn, cs;
    sincosf(pos * inv_freq[i], &sn, &cs);
    sn *= amplitude;
    cs *= amplitude;
    const float u = part[a], v = part[b];
    dst[kv_rank + a] = from_float<T>(u * cs - v * sn);
    dst[kv_rank + b] = from_float<T>(v * cs + u * sn);
  }
}

template <typename TIn, typename T>
__global__ void latent_q_store_kernel(const TIn* __restrict__ q, int splits, size_t split_stride, int num_tokens,
                                      int num_heads, int dim, int rot_dim, int kv_rank,
                                      const int* __restrict__ positions, const float* __restrict__ inv_freq,
                                      float amplitude, int interleaved, T* __restrict__ q_plain,
                                      T* __restrict__ q_full) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long warp = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  if (warp >= (long long)num_tokens * num_heads) return;
  const int t = (int)(warp / num_heads);
  const TIn* src = q + (size_t)warp * (dim + rot_dim);
  T* plain = q_plain + (size_t)warp * dim;
  for (int d = lane; d < dim; d += 32) plain[d] = from_float<T>(sum_parts(src + d, splits, split_stride));
  T* dst = q_full + (size_t)warp * (kv_rank + rot_dim) + kv_rank;
  const int half = rot_dim >> 1;
  const float pos = (float)positions[t];
  for (int i = lane; i < half; i += 32) {
    int a, b;
    pair_of(i, half, interleaved, &a, &b);
    const float u = sum_parts(src + dim + a, splits, split_stride);
    const float v = sum_parts(src + dim + b, splits, split_stride);
    float sn, cs;
    sincosf(pos * inv_freq[i], &sn, &cs);
    sn *= amplitude;
    cs *= amplitude;
    dst[a] = from_float<T>(u * cs - v * sn);
    dst[b] = from_float<T>(v * cs + u * sn);
  }
}

// blockIdx.y 0: the cache row and the gates; 1 and on: `heads_per_cta` heads' queries.  With one CTA a token
// (gridDim.y 1) it does both.
template <typename TIn, typename T>
__global__ void __launch_bounds__(128)
latent_qkv_store_kernel(const TIn* __restrict__ in, int splits, size_t split_stride, int width, int kv_rank, int rot_dim,
                        int num_heads, int dim, int row, int heads_per_cta, const float* __restrict__ kv_norm_weight,
                        float eps, const int* __restrict__ positions, const float* __restrict__ inv_freq, float amplitude,
                        int interleaved, const int* __restrict__ slots, T* __restrict__ q_plain, T* __restrict__ q_full,
                        float* __restrict__ gate, T* __restrict__ cache, int page_size, int num_pages, int* status) {
  extern __shared__ float smem[];
  const int half = rot_dim >> 1;
  float* cos_t = smem;                       // [half]
  float* sin_t = cos_t + half;               // [half]
  float* latent = sin_t + half;              // [kv_rank + rot_dim], in the CTA that writes the cache row
  __shared__ float scratch[33];
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const float pos = (float)positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, cs;
    sincosf(pos * inv_freq[i], &sn, &cs);
    sin_t[i] = amplitude * sn;
    cos_t[i] = amplitude * cs;
  }
  pdl_wait();
  __syncthreads();
  const TIn* src = in + (size_t)t * width;
  const int size = kv_rank + rot_dim;
  if (blockIdx.y == 0) {
    float squares = 0.f;
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
      const float v = sum_parts(src + i, splits, split_stride);
      latent[i] = v;
      if (i < kv_rank) squares += v * v;
    }
    if (gate) {
      const TIn* logits = src + size + num_heads * (dim + rot_dim);
      for (int h = threadIdx.x; h < num_heads; h += blockDim.x)
        gate[(size_t)t * num_heads + h] = 1.f / (1.f + expf(-sum_parts(logits + h, splits, split_stride)));
    }
    const float factor = rsqrtf(block_sum(squares, scratch) / (float)kv_rank + eps);   // has barriers: latent[] is complete
    const int slot = slots ? slots[t] : -1;
    const int page = slot >= 0 ? slot / page_size : -1;
    if (page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(status, kStatusBadPage);
    } else if (page >= 0) {
      T* dst = cache + ((size_t)page * page_size + (slot - page * page_size)) * row;
      for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) dst[i] = from_float<T>(latent[i] * factor * kv_norm_weight[i]);
      const float* part = latent + kv_rank;
      for (int i = threadIdx.x; i < half; i += blockDim.x) {
        int a, b;
        pair_of(i, half, interleaved, &a, &b);
        const float u = part[a], v = part[b], cs = cos_t[i], sn = sin_t[i];
        dst[kv_rank + a] = from_float<T>(u * cs - v * sn);
        dst[kv_rank + b] = from_float<T>(v * cs + u * sn);
      }
      for (int i = size + threadIdx.x; i < row; i += blockDim.x) dst[i] = from_float<T>(0.f);
    }
    if (gridDim.y > 1) return;
  }
  const int head0 = gridDim.y > 1 ? ((int)blockIdx.y - 1) * heads_per_cta : 0;
  const int heads = gridDim.y > 1 ? min(heads_per_cta, num_heads - head0) : num_heads;
  const TIn* queries = src + size + (size_t)head0 * (dim + rot_dim);
  if (q_plain) {
    T* plain = q_plain + ((size_t)t * num_heads + head0) * dim;
    for (int i = threadIdx.x; i < heads * dim; i += blockDim.x) {
      const int h = i / dim;
      plain[i] = from_float<T>(sum_parts(queries + i + (size_t)h * rot_dim, splits, split_stride));
    }
  }
  const int tail = row - kv_rank - rot_dim;          // zeros behind the rotated part
  const int items = half + tail;
  T* full = q_full + ((size_t)t * num_heads + head0) * row + kv_rank;
  for (int index = threadIdx.x; index < heads * items; index += blockDim.x) {
    const int h = index / items, i = index - h * items;
    T* dst = full + (size_t)h * row;
    if (i >= half) {
      dst[rot_dim + i - half] = from_float<T>(0.f);
      continue;
    }
    int a, b;
    pair_of(i, half, interleaved, &a, &b);
    const TIn* q = queries + (size_t)h * (dim + rot_dim) + dim;
    const float u = sum_parts(q + a, splits, split_stride), v = sum_parts(q + b, splits, split_stride);
    dst[a] = from_float<T>(u * cos_t[i] - v * sin_t[i]);
    dst[b] = from_float<T>(v * cos_t[i] + u * sin_t[i]);
  }
}

}  // namespace einf

using namespace einf;

// in: [T, width] (or `splits` float32 partial sums of it), of which kv_rank + rot_dim + H * (dim + rot_dim) (+ H gate
// logits, where gate [T, H] is given) elements are read; cache: [pages, 1, page_size, row]; q_plain: [T, H, dim] or null (the caller
// reads the product's own rows); q_full: [T, H, row], of which this writes the elements from kv_rank on.
extern "C" int einf_latent_qkv_store(const void* in, int in_dtype, int splits, long long split_stride, int dtype,
                                     int num_tokens, int width, int kv_rank, int rot_dim, int num_heads, int dim, int row,
                                     const float* kv_norm_weight, float eps, const int* positions, const float* inv_freq,
                                     float amplitude, int interleaved, const int* slots, void* q_plain, void* q_full,
                                     float* gate, void* cache, int page_size, int num_pages, int* status,
                                     cudaStream_t stream) {
  if (num_tokens == 0) return 0;
  if (kv_rank <= 0 || rot_dim < 0 || (rot_dim & 1) || num_heads <= 0 || dim <= 0 || row < kv_rank + rot_dim)
    return (int)cudaErrorInvalidValue;
  const size_t smem = (size_t)(kv_rank + 2 * rot_dim) * sizeof(float);
  if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
  if (width < kv_rank + rot_dim + num_heads * (dim + rot_dim) + (gate ? num_heads : 0)) return (int)cudaErrorInvalidValue;
  // a few tokens: their heads are spread over CTAs, so that the partial sums come through many SMs
  const int heads_per_cta = num_tokens >= 296 ? num_heads : max(1, 512 / (dim + rot_dim));
  const int blocks = num_tokens >= 296 ? 1 : 1 + (num_heads + heads_per_cta - 1) / heads_per_cta;
  if (blocks > 65535) return (int)cudaErrorInvalidValue;
  EINF_DISPATCH_2(in_dtype, TIn, {
    EINF_DISPATCH_2(dtype, T, {
      return (int)launch_pdl(latent_qkv_store_kernel<TIn, T>, dim3(num_tokens, blocks), dim3(128), smem, stream,
                             (const TIn*)in, splits, (size_t)split_stride, width, kv_rank, rot_dim, num_heads, dim, row,
                             heads_per_cta, kv_norm_weight, eps, positions, inv_freq, amplitude, interleaved, slots,
                             (T*)q_plain, (T*)q_full, gate, (T*)cache, page_size, num_pages, status);
    })
  })
}

// down: [T, q_rank + kv_rank + rot_dim] (or `splits` float32 partial sums of it); cache:
// [pages, 1, page_size, kv_rank + rot_dim]; q_latent_out: [T, q_rank] (q_rank may be 0).
extern "C" int einf_latent_down_store(const void* down, int in_dtype, int splits, long long split_stride, int dtype,
                                      int num_tokens, int q_rank, int kv_rank, int rot_dim,
                                      const float* q_norm_weight, const float* kv_norm_weight, float eps,
                                      const int* positions, const float* inv_freq, float amplitude, int interleaved,
                                      const int* slots, void* q_latent_out, void* cache, int page_size,
                                      int num_pages, int* status, cudaStream_t stream) {
  if (num_tokens == 0) return 0;
  if (kv_rank <= 0 || rot_dim < 0 || (rot_dim & 1) || q_rank < 0) return (int)cudaErrorInvalidValue;
  const size_t smem = (size_t)(q_rank + kv_rank + rot_dim) * sizeof(float);
  if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
  EINF_DISPATCH_2(in_dtype, TIn, {
    EINF_DISPATCH_2(dtype, T, {
      return (int)launch_pdl(latent_down_store_kernel<TIn, T>, num_tokens, 256, smem, stream, (const TIn*)down, splits,
                             (size_t)split_stride, q_rank, kv_rank, rot_dim, q_norm_weight, kv_norm_weight, eps,
                             positions, inv_freq, amplitude, interleaved, slots, (T*)q_latent_out, (T*)cache, page_size,
                             num_pages, status);
    })
  })
}

// q: [T, H * (dim + rot_dim)] (or partial sums); q_plain: [T, H, dim]; q_full: [T, H, kv_rank + rot_dim],
// of which this writes the last rot_dim elements of every head.
extern "C" int einf_latent_q_store(const void* q, int in_dtype, int splits, long long split_stride, int dtype,
                                   int num_tokens, int num_heads, int dim, int rot_dim, int kv_rank,
                                   const int* positions, const float* inv_freq, float amplitude, int interleaved, void* q_plain,
                                   void* q_full, cudaStream_t stream) {
  if (num_tokens == 0) return 0;
  const long long warps = (long long)num_tokens * num_heads;
  const int threads = 128;
  const long long blocks = (warps * 32 + threads - 1) / threads;
  if (blocks >= (1ll << 31) || (rot_dim & 1)) return (int)cudaErrorInvalidValue;
  EINF_DISPATCH_2(in_dtype, TIn, {
    EINF_DISPATCH_2(dtype, T, {
      return (int)launch_pdl(latent_q_store_kernel<TIn, T>, (int)blocks, threads, 0, stream, (const TIn*)q, splits,
                             (size_t)split_stride, num_tokens, num_heads, dim, rot_dim, kv_rank, positions, inv_freq,
                             amplitude, interleaved, (T*)q_plain, (T*)q_full);
    })
  })
}
