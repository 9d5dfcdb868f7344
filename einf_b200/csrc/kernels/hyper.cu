// Residual streams that sublayers read and write through vectors of their own, and the norm in
// front of a sublayer, in one pass over a token's row of every stream (all of it 32-bit):
//
//   the write of the sublayer before   x'_t = sum_s mix[s, t] x_s + write[t] * y
//   what the next sublayer reads       u = sum_t read[t] x'_t
//   its norm                           out = norm(u) * weight (+ bias), RMS or layer norm
//
// y is a [T, H] matrix (float or bfloat16), the float partial sums [S, T, H] of a split-K product,
// or absent.  Without `mix` the one stream is plain: x' = x + y.  Without `read` the streams are
// added up (the end of the model).  `source_stride` 0 means that all streams are still equal and
// stored once (the embedding output).  With `dest` the x'_t are stored; it may be the source
// itself.  With `rows`, output row r is computed from row rows[r] and nothing is stored.
//
//   layer norm   (u - mean) / sqrt(mean((u - mean)^2) + eps), the two means one after the other
//   RMS norm     u / sqrt(mean(u^2) + eps)
//
// A row is computed from itself alone, in an order that depends on the sizes only.
//
// Three kernels: a warp per row with u in registers (many rows, no partial sums), a CTA per row
// with a float4 of u per thread and all partial sums in flight together (a decode step's few
// rows), and a CTA per row with u in shared memory (any width).
#include "common.cuh"

namespace einf {

constexpr int kMaxStreams = 16;

struct HyperParams {
  const void* y;
  long long y_stride;
  const float* source;
  long long source_stride;      // between two streams; 0: one row stands for all of them
  const float* mix;             // [streams, streams], from the first index to the second
  const float* write;           // [streams]
  const float* read;            // [streams] or null: ones
  float* dest;
  long long dest_stride;
  const float* weight;
  const float* bias;            // null: none
  void* out;
  const int* rows;
  int y_splits, streams, num_rows, hidden, centre;
  float eps;
};

// The coefficients of a launch in registers: S streams at compile time, or up to kMaxStreams.
template <int S>
struct Coefficients {
  float mix[S][S], write[S], read[S];
  __device__ __forceinline__ void load(const HyperParams& p) {
#pragma unroll
    for (int t = 0; t < S; ++t) {
      const bool live = t < p.streams;
#pragma unroll
      for (int s = 0; s < S; ++s)
        mix[s][t] = (live && s < p.streams) ? (p.mix ? p.mix[s * p.streams + t] : (s == t ? 1.f : 0.f)) : 0.f;
      write[t] = live ? (p.mix ? p.write[t] : 1.f) : 0.f;
      read[t] = live ? (p.read ? p.read[t] : 1.f) : 0.f;
    }
  }
};

__device__ __forceinline__ float4 hyper_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 hyper_load4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void hyper_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void hyper_store4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<const uint32_t*>(&a);
  raw.y = *reinterpret_cast<const uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = raw;
}
__device__ __forceinline__ void fma4(float4& acc, float f, const float4& v) {
  acc.x = fmaf(f, v.x, acc.x);
  acc.y = fmaf(f, v.y, acc.y);
  acc.z = fmaf(f, v.z, acc.z);
  acc.w = fmaf(f, v.w, acc.w);
}
__device__ __forceinline__ float sum4(const float4& v) { return (v.x + v.y) + (v.z + v.w); }
__device__ __forceinline__ float square4(const float4& v, float mean) {
  const float a = v.x - mean, b = v.y - mean, c = v.z - mean, d = v.w - mean;
  return (a * a + b * b) + (c * c + d * d);
}

// Mix four elements of every stream, store them, and return what the sublayer reads of them.
template <int S>
__device__ __forceinline__ float4 mix_and_read(const Coefficients<S>& c, const float4 (&x)[S], const float4& y, bool adds,
                                               float* dest, long long dest_stride, int streams) {
  float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int t = 0; t < S; ++t) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int s = 0; s < S; ++s) fma4(v, c.mix[s][t], x[s]);
    if (adds) fma4(v, c.write[t], y);
    if (dest && t < streams) hyper_store4(dest + (long long)t * dest_stride, v);
    fma4(u, c.read[t], v);
  }
  return u;
}

__device__ __forceinline__ float4 scale4(const float4& u, float mean, float factor, const float4& w, const float4& b) {
  return make_float4(fmaf((u.x - mean) * factor, w.x, b.x), fmaf((u.y - mean) * factor, w.y, b.y),
                     fmaf((u.z - mean) * factor, w.z, b.z), fmaf((u.w - mean) * factor, w.w, b.w));
}

// One warp per row, kVec float4 of u per lane (hidden <= 128 * kVec, a multiple of 4).  The rows of kChunk
// vectors of all streams are in flight at a time (a store into a stream may not pass a later load).
template <typename TY, typename TOut, int S, int kVec>
__global__ void __launch_bounds__(128)
hyper_norm_warp_kernel(const __grid_constant__ HyperParams p) {
  constexpr int kChunk = kVec < 4 ? kVec : (S >= 4 ? 2 : 4);
  pdl_launch_dependents();
  Coefficients<S> c;
  c.load(p);
  pdl_wait();
  const int r = (int)((blockIdx.x * blockDim.x + threadIdx.x) >> 5);
  const int lane = threadIdx.x & 31;
  if (r >= p.num_rows) return;
  const int row = p.rows ? p.rows[r] : r;
  const size_t base = (size_t)row * p.hidden;
  const TY* y = p.y ? (const TY*)p.y + base : nullptr;
  float* dest = p.dest ? p.dest + base : nullptr;
  float4 u[kVec];
  float total = 0.f;
#pragma unroll
  for (int j0 = 0; j0 < kVec; j0 += kChunk) {
    float4 x[kChunk][S], add[kChunk];
#pragma unroll
    for (int j = 0; j < kChunk; ++j) {
      // an index past the row is clamped: its values are not used
      const int i = min(((j0 + j) * 32 + lane) * 4, p.hidden - 4);
#pragma unroll
      for (int s = 0; s < S; ++s)
        x[j][s] = hyper_load4(p.source + (s < p.streams ? (long long)s * p.source_stride : 0) + base + i);
      add[j] = y ? hyper_load4(y + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < kChunk; ++j) {
      const int i = ((j0 + j) * 32 + lane) * 4;
      u[j0 + j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < p.hidden) {
        u[j0 + j] = mix_and_read<S>(c, x[j], add[j], y != nullptr, dest ? dest + i : nullptr, p.dest_stride, p.streams);
        total += sum4(u[j0 + j]);
      }
    }
  }
  const float mean = p.centre ? warp_sum(total) / (float)p.hidden : 0.f;
  float squares = 0.f;
#pragma unroll
  for (int j = 0; j < kVec; ++j)
    if ((j * 32 + lane) * 4 < p.hidden) squares += square4(u[j], mean);
  const float factor = rsqrtf(warp_sum(squares) / (float)p.hidden + p.eps);
  TOut* out = (TOut*)p.out + (size_t)r * p.hidden;
#pragma unroll
  for (int j = 0; j < kVec; ++j) {
    const int i = (j * 32 + lane) * 4;
    if (i < p.hidden) {
      const float4 b = p.bias ? hyper_load4(p.bias + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      hyper_store4(out + i, scale4(u[j], mean, factor, hyper_load4(p.weight + i), b));
    }
  }
}

// One CTA per row, one float4 of u per thread (hidden <= 4 * kThreads, a multiple of 4): every load of a thread goes
// out before the first is used, the partial sums a batch at a time (sixteen where a thread has the registers).
template <typename TY, typename TOut, int S, int kThreads>
__global__ void __launch_bounds__(kThreads)
hyper_norm_row_kernel(const __grid_constant__ HyperParams p) {
  constexpr int kHyperBatch = kThreads <= 512 ? 16 : 8;
  __shared__ float sums[2][32];
  pdl_launch_dependents();
  const int i = (int)threadIdx.x * 4;
  const bool live = i < p.hidden;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const float4 w = live ? hyper_load4(p.weight + i) : zero;
  const float4 b = live && p.bias ? hyper_load4(p.bias + i) : zero;
  Coefficients<S> c;
  c.load(p);
  const int r = blockIdx.x;
  const int row = p.rows ? p.rows[r] : r;
  const size_t base = (size_t)row * p.hidden + i;
  pdl_wait();
  float4 u = zero;
  if (live) {
    float4 x[S];
#pragma unroll
    for (int s = 0; s < S; ++s) x[s] = hyper_load4(p.source + (s < p.streams ? (long long)s * p.source_stride : 0) + base);
    float4 add = zero;
    if (p.y) {
      const TY* y = (const TY*)p.y + base;
      for (int k = 0; k < p.y_splits; k += kHyperBatch) {
        float4 t[kHyperBatch];
#pragma unroll
        for (int e = 0; e < kHyperBatch; ++e) t[e] = hyper_load4(y + (long long)min(k + e, p.y_splits - 1) * p.y_stride);
#pragma unroll
        for (int e = 0; e < kHyperBatch; ++e)
          if (k + e < p.y_splits) fma4(add, 1.f, t[e]);
      }
    }
    u = mix_and_read<S>(c, x, add, p.y != nullptr, p.dest ? p.dest + base : nullptr, p.dest_stride, p.streams);
  }
  float mean = 0.f;
  if (p.centre) {
    const float total = warp_sum(sum4(u));
    if (lane == 0) sums[0][warp] = total;
    __syncthreads();
    mean = warp_sum(lane < warps ? sums[0][lane] : 0.f) / (float)p.hidden;   // the same order in every warp
  }
  const float squares = warp_sum(live ? square4(u, mean) : 0.f);
  if (lane == 0) sums[1][warp] = squares;
  __syncthreads();
  const float factor = rsqrtf(warp_sum(lane < warps ? sums[1][lane] : 0.f) / (float)p.hidden + p.eps);
  if (live) hyper_store4((TOut*)p.out + (size_t)r * p.hidden + i, scale4(u, mean, factor, w, b));
}

// One CTA per row, u in shared memory: any width, any number of streams.
template <typename TY, typename TOut, int S>
__global__ void __launch_bounds__(512)
hyper_norm_kernel(const __grid_constant__ HyperParams p) {
  extern __shared__ float smem[];
  float* u_row = smem;                        // [hidden]
  float* scratch = smem + p.hidden;           // [33]
  float* mix = scratch + 33;                  // [streams][streams], [streams] written, [streams] read
  float* write = mix + S * S;
  float* read = write + S;
  pdl_launch_dependents();
  const int streams = p.streams;
  for (int k = threadIdx.x; k < streams * streams; k += blockDim.x)
    mix[k] = p.mix ? p.mix[k] : (k / streams == k % streams ? 1.f : 0.f);
  for (int k = threadIdx.x; k < streams; k += blockDim.x) {
    write[k] = p.mix ? p.write[k] : 1.f;
    read[k] = p.read ? p.read[k] : 1.f;
  }
  __syncthreads();
  pdl_wait();
  const int r = blockIdx.x;
  const int row = p.rows ? p.rows[r] : r;
  const size_t base = (size_t)row * p.hidden;
  float total = 0.f;
  for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
    float x[S];
#pragma unroll
    for (int s = 0; s < S; ++s) x[s] = s < streams ? p.source[(long long)s * p.source_stride + base + i] : 0.f;
    float y = 0.f;
    if (p.y) {
      const TY* q = (const TY*)p.y + base + i;
      int k = 0;
      for (; k + 8 <= p.y_splits; k += 8) {
        float t[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) t[e] = to_float(q[(long long)(k + e) * p.y_stride]);
#pragma unroll
        for (int e = 0; e < 8; ++e) y += t[e];
      }
      for (; k < p.y_splits; ++k) y += to_float(q[(long long)k * p.y_stride]);
    }
    float u = 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) {
      if (t < streams) {
        float v = 0.f;
#pragma unroll
        for (int s = 0; s < S; ++s)
          if (s < streams) v = fmaf(mix[s * streams + t], x[s], v);
        if (p.y) v = fmaf(write[t], y, v);
        if (p.dest) p.dest[(long long)t * p.dest_stride + base + i] = v;
        u = fmaf(read[t], v, u);
      }
    }
    u_row[i] = u;
    total += u;
  }
  const float mean = p.centre ? block_sum(total, scratch) / (float)p.hidden : 0.f;
  float squares = 0.f;
  for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
    const float d = u_row[i] - mean;
    squares = fmaf(d, d, squares);
  }
  const float factor = rsqrtf(block_sum(squares, scratch) / (float)p.hidden + p.eps);
  TOut* out = (TOut*)p.out + (size_t)r * p.hidden;
  for (int i = threadIdx.x; i < p.hidden; i += blockDim.x)
    out[i] = from_float<TOut>(fmaf((u_row[i] - mean) * factor, p.weight[i], p.bias ? p.bias[i] : 0.f));
}

template <typename TY, typename TOut, int S>
int launch_hyper(const HyperParams& p, bool vectors, cudaStream_t stream) {
  if (vectors && S <= 4 && p.y_splits == 1 && p.num_rows > 128 && p.hidden <= 4096) {
    constexpr int kS = S <= 4 ? S : 1;      // larger counts never come here
    const int warps = 4, blocks = (p.num_rows + warps - 1) / warps;
    if (p.hidden <= 512) return (int)launch_pdl(hyper_norm_warp_kernel<TY, TOut, kS, 4>, blocks, warps * 32, 0, stream, p);
    if (p.hidden <= 1024) return (int)launch_pdl(hyper_norm_warp_kernel<TY, TOut, kS, 8>, blocks, warps * 32, 0, stream, p);
    if (p.hidden <= 2048) return (int)launch_pdl(hyper_norm_warp_kernel<TY, TOut, kS, 16>, blocks, warps * 32, 0, stream, p);
    return (int)launch_pdl(hyper_norm_warp_kernel<TY, TOut, kS, 32>, blocks, warps * 32, 0, stream, p);
  }
  if (vectors && S <= 4 && p.hidden <= 4096) {
    constexpr int kS = S <= 4 ? S : 1;
    const int threads = (p.hidden / 4 + 31) / 32 * 32;
    if (threads <= 512)
      return (int)launch_pdl(hyper_norm_row_kernel<TY, TOut, kS, 512>, p.num_rows, threads, 0, stream, p);
    return (int)launch_pdl(hyper_norm_row_kernel<TY, TOut, kS, 1024>, p.num_rows, threads, 0, stream, p);
  }
  const size_t smem = (size_t)(p.hidden + 33 + S * S + 2 * S) * sizeof(float);
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  auto kernel = hyper_norm_kernel<TY, TOut, S>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  int threads = 64;
  while (threads < p.hidden && threads < 512) threads <<= 1;
  return (int)launch_pdl(kernel, p.num_rows, threads, smem, stream, p);
}

}  // namespace einf

using namespace einf;

// y: null, [T, hidden] or y_splits float32 partial sums of it; source, dest: float32 rows of `hidden`, the streams
// source_stride / dest_stride elements apart; out: [num_rows, hidden].
extern "C" int einf_hyper_norm(const void* y, int y_dtype, int y_splits, long long y_stride, const float* source,
                               long long source_stride, int streams, const float* mix, const float* write,
                               const float* read, float* dest, long long dest_stride, const float* weight,
                               const float* bias, int centre, float eps, void* out, int out_dtype, const int* rows,
                               int num_rows, int hidden, cudaStream_t stream) {
  if (num_rows == 0) return 0;
  if (streams < 1 || streams > kMaxStreams || hidden < 1 || y_splits < 1 || (!mix && streams != 1 && y) || (mix && !write) ||
      (rows && dest))
    return (int)cudaErrorInvalidValue;
  HyperParams p = {y, y_stride, source, source_stride, mix, write, read, dest, dest_stride, weight, bias, out, rows,
                   y_splits, streams, num_rows, hidden, centre, eps};
  auto aligned = [](const void* q) { return ((uintptr_t)q & 15) == 0; };
  const bool vectors = hidden % 4 == 0 && aligned(y) && aligned(source) && aligned(dest) && aligned(weight) &&
                       aligned(bias) && aligned(out) && y_stride % 4 == 0 && source_stride % 4 == 0 && dest_stride % 4 == 0;
  EINF_DISPATCH_2(y_dtype, TY, {
    EINF_DISPATCH_2(out_dtype, TOut, {
      if (streams == 1) return launch_hyper<TY, TOut, 1>(p, vectors, stream);
      if (streams == 2) return launch_hyper<TY, TOut, 2>(p, vectors, stream);
      if (streams <= 4) return launch_hyper<TY, TOut, 4>(p, vectors, stream);
      return launch_hyper<TY, TOut, kMaxStreams>(p, vectors, stream);
    })
  })
}
