// Between an attention layer's product for queries, keys and values and its attention kernel, for
// layers that convolve the projections over time: bias, a causal convolution of `taps` taps on every
// channel, rotation of the convolved queries and keys, the paged write of keys and values.
//
// A row of the product is [H query heads of key_size | G key heads | G value heads of value_size | gate],
// of which the channels in front of the gate are convolved:
//   u_t = product[t] + bias,   y_t = sum_j w[:, j] u_(t - taps + 1 + j)
// over the tokens of t's request, with the request's state (its last taps - 1 inputs u, oldest first,
// floats, zeros at the sequence's start) in front of the first token of the step.  The first 2n
// dimensions of every query and key head are then rotated by the token's position: pair i is (i, i + n)
// or, interleaved, (2i, 2i + 1); (u, v) -> (u cos a - v sin a, v cos a + u sin a), a = position * inv_freq[i].
// Arithmetic is 32-bit; a value is rounded once, when it is stored.  A token's result depends on its own
// request alone.  G = 0: a layer that reads another layer's keys and values; the row holds queries (and gate).
#include "common.cuh"

namespace einf {

constexpr int kMaxTaps = 16;

template <typename TIn>
__device__ __forceinline__ float sum_parts(const TIn* p, int splits, long long stride) {
  if (splits == 1) return to_float(*p);
  constexpr int kBatch = 16;             // the partial sums sit in L2: keep all of a batch's loads in flight
  float v = 0.f;
  for (int s0 = 0; s0 < splits; s0 += kBatch) {
    float part[kBatch];
#pragma unroll
    for (int e = 0; e < kBatch; ++e) part[e] = to_float(p[(size_t)min(s0 + e, splits - 1) * stride]);
#pragma unroll
    for (int e = 0; e < kBatch; ++e)
      if (s0 + e < splits) v += part[e];
  }
  return v;
}

struct ConvStore {
  int splits, width, channels, taps;
  long long split_stride;
  const float* bias;          // [channels] or null
  const float* weight;        // [channels, taps], or null: no convolution (taps 1)
  float* state;               // [slots][taps - 1, channels]
  long long state_stride;
  int num_slots;
  const int* seq_of_token;
  const int* q_start;
  const int* state_slots;
  const int* slots;           // cache slot of every token, or null: no keys and values are written
  int num_tokens, num_heads, num_kv_heads, key_size, value_size, page_size, num_pages;
  const int* positions;
  const float* inv_freq;
  int pairs, interleaved;
  int single_tokens;          // every request brings one token: the state moves on in the same launch
  int* status;
};

__device__ __forceinline__ float* request_state(const ConvStore& p, int request) {
  const int slot = p.state_slots[request];
  return p.state && slot >= 0 && slot < p.num_slots ? p.state + (long long)slot * p.state_stride : nullptr;
}

// Page and offset of a token's cache slot; false: not written.
__device__ __forceinline__ bool cache_place(const ConvStore& p, int t, int& page, int& offset, bool reports) {
  const int slot = p.slots ? p.slots[t] : -1;
  if (slot < 0) return false;
  page = slot / p.page_size;
  offset = slot - page * p.page_size;
  if (page >= p.num_pages) {
    if (reports) atomicOr(p.status, kStatusBadPage);
    return false;
  }
  return true;
}

// ---------------------------------------------------------------------------
// Any sizes, partial sums, single tokens: a CTA per (token, head), a thread per element.  Behind the heads
// come the gate's pieces of value_size columns, which are only added up and copied out.
// ---------------------------------------------------------------------------
template <typename TIn, typename T>
__global__ void qkv_conv_head_kernel(const TIn* __restrict__ qkv, const __grid_constant__ ConvStore p, T* __restrict__ q_out,
                                     T* __restrict__ k_cache, T* __restrict__ v_cache, T* __restrict__ gate_out) {
  __shared__ float line[256];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, item = blockIdx.y, d = threadIdx.x;
  const int heads = p.num_heads, groups = p.num_kv_heads;
  const TIn* row = qkv + (size_t)t * p.width;
  if (item >= heads + 2 * groups) {
    const int at = (item - heads - 2 * groups) * p.value_size + d;
    if (d < p.value_size)
      gate_out[(size_t)t * heads * p.value_size + at] = from_float<T>(sum_parts(row + p.channels + at, p.splits, p.split_stride));
    return;
  }
  const bool is_value = item >= heads + groups;
  const int size = is_value ? p.value_size : p.key_size;
  const int c = (is_value ? (heads + groups) * p.key_size + (item - heads - groups) * p.value_size : item * p.key_size) + d;
  const int r = p.seq_of_token[t];
  float v = 0.f;
  if (d < size) {
    const float bias = p.bias ? p.bias[c] : 0.f;
    v = sum_parts(row + c, p.splits, p.split_stride) + bias;
    if (p.weight) {
      const float* w = p.weight + (size_t)c * p.taps;
      const int keep = p.taps - 1;
      float* state = keep > 0 ? request_state(p, r) : nullptr;
      float acc = 0.f;
      if (p.single_tokens) {
        float old[kMaxTaps];
#pragma unroll
        for (int j = 0; j < kMaxTaps; ++j)
          if (j < keep) old[j] = state ? state[(size_t)j * p.channels + c] : 0.f;
#pragma unroll
        for (int j = 0; j < kMaxTaps; ++j)
          if (j < keep) acc = fmaf(w[j], old[j], acc);
        if (state) {
#pragma unroll
          for (int j = 0; j < kMaxTaps; ++j)
            if (j + 1 < keep) state[(size_t)j * p.channels + c] = old[j + 1];
          state[(size_t)(keep - 1) * p.channels + c] = v;
        }
      } else {
        const int first = p.q_start[r];
        for (int j = 0; j < keep; ++j) {
          const int src = t - keep + j;
          float u;
          if (src >= first) u = sum_parts(qkv + (size_t)src * p.width + c, p.splits, p.split_stride) + bias;
          else u = state ? state[(size_t)(keep - (first - src)) * p.channels + c] : 0.f;
          acc = fmaf(w[j], u, acc);
        }
      }
      v = fmaf(w[keep], v, acc);
    }
  }
  T* dst;
  if (item < heads) {
    dst = q_out + ((size_t)t * heads + item) * p.key_size;
  } else {
    int page = 0, offset = 0;
    if (!cache_place(p, t, page, offset, d == 0)) return;          // the same for the whole CTA
    dst = is_value ? v_cache + (((size_t)page * groups + (item - heads - groups)) * p.page_size + offset) * p.value_size
                   : k_cache + (((size_t)page * groups + (item - heads)) * p.page_size + offset) * p.key_size;
  }
  if (!is_value && p.pairs > 0) {
    line[d] = v;
    __syncthreads();
    if (d < 2 * p.pairs) {
      int pair, other;
      bool leads;
      if (p.interleaved) {
        pair = d >> 1; leads = (d & 1) == 0; other = d ^ 1;
      } else {
        leads = d < p.pairs; pair = leads ? d : d - p.pairs; other = leads ? d + p.pairs : pair;
      }
      float sn, cs;
      sincosf((float)p.positions[t] * p.inv_freq[pair], &sn, &cs);
      v = leads ? v * cs - line[other] * sn : v * cs + line[other] * sn;
    }
  }
  if (d < size) dst[d] = from_float<T>(v);
}

// ---------------------------------------------------------------------------
// Prompt sizes: bfloat16 rows, pairs interleaved (or no rotation), everything in whole pieces of eight
// elements.  A thread has one piece of the row for a run of consecutive tokens: it reads every row's
// piece once (16 bytes) and carries the taps - 1 inputs before it in registers; where a request starts it
// takes them from the request's state.  The first taps - 1 tokens of a request, the only ones that see
// the state, all belong to the run in which the request starts (a run may so reach up to taps - 2 tokens
// beyond its end, and the next one leaves them out); the thread that has read the state there moves it
// on in the same breath, since the request's last inputs are rows of the product.  The run's angles,
// requests and cache places are made once per CTA, from the step's inputs alone, while the product
// before this kernel still runs.
// ---------------------------------------------------------------------------
constexpr int kRun = 8;                  // rows whose loads are in flight together
constexpr int kPieceThreads = 256;       // at most

template <int kTaps>
__global__ void __launch_bounds__(kPieceThreads, 2)
qkv_conv_piece_kernel(const __nv_bfloat16* __restrict__ qkv, const __grid_constant__ ConvStore p,
                      __nv_bfloat16* __restrict__ q_out, __nv_bfloat16* __restrict__ k_cache,
                      __nv_bfloat16* __restrict__ v_cache) {
  constexpr int kKeep = kTaps - 1, kExtra = kKeep > 1 ? kKeep - 1 : 0;
  extern __shared__ float2 angles[];     // [kRun + kExtra][pairs]: cosine, sine
  // request_of: -1 for a token of another run
  __shared__ int request_of[kRun + kExtra], first_of[kRun + kExtra], page_of[kRun + kExtra], offset_of[kRun + kExtra];
  pdl_launch_dependents();
  const int t0 = blockIdx.y * kRun, count = min(kRun + kExtra, p.num_tokens - t0);
  for (int s = threadIdx.x; s < count; s += blockDim.x) {
    const int t = t0 + s, r = p.seq_of_token[t], first = p.q_start[r];
    const bool sees_state = t - first < kKeep;
    const bool mine = s < kRun ? !sees_state || first >= t0 : sees_state && first < t0 + kRun;
    request_of[s] = mine ? r : -1;
    first_of[s] = first;
    int page = 0, offset = 0;
    page_of[s] = cache_place(p, t, page, offset, false) ? page : -1;
    offset_of[s] = offset;
  }
  for (int i = threadIdx.x; i < count * p.pairs; i += blockDim.x) {
    const int s = i / p.pairs, pair = i - s * p.pairs;
    float sn, cs;
    sincosf((float)p.positions[t0 + s] * p.inv_freq[pair], &sn, &cs);
    angles[i] = make_float2(cs, sn);
  }
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  const bool live = c < p.channels;
  float w[kTaps][8], bias[8];            // weights: no kernel of the step writes them
  if (live) {
#pragma unroll
    for (int e = 0; e < 8; e += 4) {
      const float4 b = p.bias ? *reinterpret_cast<const float4*>(p.bias + c + e) : make_float4(0.f, 0.f, 0.f, 0.f);
      bias[e] = b.x; bias[e + 1] = b.y; bias[e + 2] = b.z; bias[e + 3] = b.w;
    }
    // the taps of eight channels lie one after the other: whole float4s
#pragma unroll
    for (int i = 0; i < 2 * kTaps; ++i) {
      const float4 v = p.weight ? *reinterpret_cast<const float4*>(p.weight + (size_t)c * kTaps + 4 * i)
                                : make_float4(1.f, 1.f, 1.f, 1.f);
      const float part[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) w[(4 * i + j) % kTaps][(4 * i + j) / kTaps] = part[j];
    }
  }
  __syncthreads();
  pdl_wait();
  if (p.slots && blockIdx.x == 0 && threadIdx.x < count && page_of[threadIdx.x] < 0 && p.slots[t0 + threadIdx.x] >= 0)
    atomicOr(p.status, kStatusBadPage);
  if (!live) return;
  const int queries = p.num_heads * p.key_size, keys = p.num_kv_heads * p.key_size;
  const bool is_query = c < queries, is_value = c >= queries + keys;
  const int local = is_query ? c : (is_value ? c - queries - keys : c - queries);
  const int size = is_value ? p.value_size : p.key_size;
  const int head = local / size, d = local - head * size;
  const bool rotates = !is_value && d < 2 * p.pairs;

  float past[kKeep > 0 ? kKeep : 1][8];
  auto load_row = [&](int t) { return *reinterpret_cast<const uint4*>(qkv + (size_t)t * p.width + c); };
  auto unpack = [&](const uint4& raw, float (&u)[8]) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(h[e]);
      u[2 * e] = f.x + bias[2 * e];
      u[2 * e + 1] = f.y + bias[2 * e + 1];
    }
  };
  // The inputs before token t of request r: rows of the step, or, for the request's first token, its state, whose
  // place then gets the request's last inputs (a portion shorter than that keeps the tail of the old ones in front).
  auto enter = [&](int t, int r, int first) {
    if (t > first) {                     // the run starts inside the request, where no token sees the state
#pragma unroll
      for (int j = 0; j < kKeep; ++j) unpack(load_row(t - kKeep + j), past[j]);
      return;
    }
    float* state = request_state(p, r);
#pragma unroll
    for (int j = 0; j < kKeep; ++j)
#pragma unroll
      for (int e = 0; e < 8; e += 4) {
        const float4 v = state ? *reinterpret_cast<const float4*>(state + (size_t)j * p.channels + c + e)
                               : make_float4(0.f, 0.f, 0.f, 0.f);
        past[j][e] = v.x; past[j][e + 1] = v.y; past[j][e + 2] = v.z; past[j][e + 3] = v.w;
      }
    if (!state) return;
    const int length = p.q_start[r + 1] - first;
#pragma unroll
    for (int j = 0; j < kKeep; ++j) {
      const int rel = length - kKeep + j;
      float4* row = reinterpret_cast<float4*>(state + (size_t)j * p.channels + c);
      if (rel >= 0) {
        float fresh[8];
        unpack(load_row(first + rel), fresh);
        row[0] = make_float4(fresh[0], fresh[1], fresh[2], fresh[3]);
        row[1] = make_float4(fresh[4], fresh[5], fresh[6], fresh[7]);
      } else {                           // a later row, not yet written
        const float4* old = reinterpret_cast<const float4*>(state + (size_t)(j + length) * p.channels + c);
        row[0] = old[0];
        row[1] = old[1];
      }
    }
  };
  int request = -1;
  auto step = [&](int s, const uint4& raw) {
    const int t = t0 + s, r = request_of[s];
    if (r < 0) return;
    if (kKeep > 0 && r != request) enter(t, r, first_of[s]);
    request = r;
    float u[8], y[8];
    unpack(raw, u);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < kKeep; ++j) acc = fmaf(w[j][e], past[j][e], acc);
      y[e] = fmaf(w[kKeep][e], u[e], acc);
#pragma unroll
      for (int j = 0; j + 1 < kKeep; ++j) past[j][e] = past[j + 1][e];
      if (kKeep > 0) past[kKeep > 0 ? kKeep - 1 : 0][e] = u[e];
    }
    if (rotates) {
      const float2* a = angles + s * p.pairs + (d >> 1);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 cs = a[e];
        const float even = y[2 * e], odd = y[2 * e + 1];
        y[2 * e] = even * cs.x - odd * cs.y;
        y[2 * e + 1] = odd * cs.x + even * cs.y;
      }
    }
    __nv_bfloat16* dst;
    if (is_query) {
      dst = q_out + (size_t)t * queries + c;
    } else {
      if (page_of[s] < 0) return;
      dst = (is_value ? v_cache : k_cache) +
            (((size_t)page_of[s] * p.num_kv_heads + head) * p.page_size + offset_of[s]) * size + d;
    }
    uint4 packed;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
    for (int e = 0; e < 4; ++e) h[e] = __floats2bfloat162_rn(y[2 * e], y[2 * e + 1]);
    *reinterpret_cast<uint4*>(dst) = packed;
  };
  uint4 raw[kRun];
#pragma unroll
  for (int s = 0; s < kRun; ++s) raw[s] = load_row(t0 + min(s, count - 1));
#pragma unroll
  for (int s = 0; s < kRun; ++s)
    if (s < count) step(s, raw[s]);
#pragma unroll 1
  for (int s = kRun; s < count; ++s)
    if (request_of[s] >= 0) step(s, load_row(t0 + s));
}

// After the head-by-head kernel a request's last taps - 1 inputs become its state (a portion shorter than
// that keeps the tail of the old state in front).  One thread per (request, channel).
template <typename TIn>
__global__ void qkv_conv_state_kernel(const TIn* __restrict__ qkv, const __grid_constant__ ConvStore p) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= p.channels) return;
  float* state = request_state(p, r);
  const int first = p.q_start[r], count = p.q_start[r + 1] - first;
  if (!state || count <= 0) return;
  const int keep = p.taps - 1;
  const float bias = p.bias ? p.bias[c] : 0.f;
  float fresh[kMaxTaps];
#pragma unroll
  for (int u = 0; u < kMaxTaps; ++u) {
    if (u < keep) {
      const int rel = count - keep + u;
      fresh[u] = rel >= 0 ? sum_parts(qkv + (size_t)(first + rel) * p.width + c, p.splits, p.split_stride) + bias
                          : state[(size_t)(u + count) * p.channels + c];
    }
  }
#pragma unroll
  for (int u = 0; u < kMaxTaps; ++u)
    if (u < keep) state[(size_t)u * p.channels + c] = fresh[u];
}

}  // namespace einf

using namespace einf;

extern "C" int einf_qkv_conv_store(const void* qkv, int in_dtype, int splits, long long split_stride, int width, int dtype,
                                   const float* bias, const float* conv_weight, int taps, float* conv_state,
                                   long long state_stride, int num_slots, const int* seq_of_token, const int* q_start,
                                   const int* state_slots, int num_requests, const int* slots, void* q_out, void* k_cache,
                                   void* v_cache, int num_tokens, int num_heads, int num_kv_heads, int key_size,
                                   int value_size, int page_size, int num_pages, const int* positions,
                                   const float* inv_freq, int pairs, int interleaved, void* gate_out, int single_tokens,
                                   int* status, cudaStream_t stream) {
  if (num_tokens == 0) return 0;
  if (num_heads <= 0 || num_kv_heads < 0 || key_size <= 0 || value_size <= 0 || key_size > 256 || value_size > 256 ||
      taps < 1 || taps > kMaxTaps || pairs < 0 || 2 * pairs > key_size || (pairs > 0 && (!positions || !inv_freq)) ||
      (taps > 1 && (!conv_weight || !conv_state)) || num_requests > 65535 || (slots && page_size <= 0))
    return (int)cudaErrorInvalidValue;
  const int channels = (num_heads + num_kv_heads) * key_size + num_kv_heads * value_size;
  if (width < channels || (gate_out && width < channels + num_heads * value_size)) return (int)cudaErrorInvalidValue;
  const ConvStore p{splits < 1 ? 1 : splits, width, channels, taps, split_stride, bias, conv_weight, conv_state,
                    state_stride, num_slots, seq_of_token, q_start, state_slots, slots, num_tokens, num_heads,
                    num_kv_heads, key_size, value_size, page_size, num_pages, positions, inv_freq, pairs, interleaved,
                    single_tokens, status};
  const bool pieces = in_dtype == kBFloat16 && dtype == kBFloat16 && p.splits == 1 && !single_tokens && !gate_out &&
                      num_tokens >= 32 && taps <= 4 && key_size % 8 == 0 && value_size % 8 == 0 && width % 8 == 0 &&
                      pairs % 4 == 0 && (interleaved || pairs == 0) && num_tokens <= 65535 * kRun &&
                      (taps == 1 || state_stride % 4 == 0) &&
                      (((uintptr_t)qkv | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)bias |
                        (uintptr_t)conv_weight | (uintptr_t)conv_state) & 15) == 0;
  cudaError_t e = cudaSuccess;
  if (pieces) {
    // equal shares of a row's pieces, so that few threads are left over
    const int shares = (channels / 8 + kPieceThreads - 1) / kPieceThreads;
    const int threads = ((channels / 8 + shares - 1) / shares + 31) / 32 * 32;
    const dim3 grid(shares, (num_tokens + kRun - 1) / kRun);
#define EINF_PIECES(TAPS)                                                                                        \
  e = launch_pdl(qkv_conv_piece_kernel<TAPS>, grid, threads, (size_t)(kRun + TAPS) * pairs * sizeof(float2),     \
                 stream, (const __nv_bfloat16*)qkv, p, (__nv_bfloat16*)q_out, (__nv_bfloat16*)k_cache,           \
                 (__nv_bfloat16*)v_cache)
    if (taps == 1) EINF_PIECES(1);
    else if (taps == 2) EINF_PIECES(2);
    else if (taps == 3) EINF_PIECES(3);
    else EINF_PIECES(4);
#undef EINF_PIECES
    return (int)e;
  }
  {
    const int items = num_heads + 2 * num_kv_heads + (gate_out ? num_heads : 0);
    if (items > 65535) return (int)cudaErrorInvalidValue;
    const int largest = key_size > value_size ? key_size : value_size;
    const int threads = (largest + 31) / 32 * 32;
    EINF_DISPATCH_2(in_dtype, TIn, {
      EINF_DISPATCH_2(dtype, T, {
        e = launch_pdl(qkv_conv_head_kernel<TIn, T>, dim3(num_tokens, items), threads, 0, stream, (const TIn*)qkv, p,
                       (T*)q_out, (T*)k_cache, (T*)v_cache, (T*)gate_out);
      })
    })
  }
  if (e != cudaSuccess || taps == 1 || single_tokens) return (int)e;
  const dim3 grid((channels + 127) / 128, num_requests);
  EINF_DISPATCH_2(in_dtype, TIn, {
    return (int)launch_pdl(qkv_conv_state_kernel<TIn>, grid, 128, 0, stream, (const TIn*)qkv, p);
  })
}
