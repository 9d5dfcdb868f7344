// Causal attention over cached rows that all query heads share and whose leading elements are the values
// (a latent cache), on the fifth-generation tensor cores, for rows of any multiple of 64 elements up to 640.
//
// With one key/value head every (token, head) pair is a query row over the same keys, so the packed queries
// [tokens * heads, row] are one matrix and a CTA takes 128 consecutive rows of it: all heads of a few tokens
// (128 / heads of them), which see nearly the same keys.  A short window therefore costs what it should (a tile
// of 128 tokens of one head would walk window + 128 keys, this one window + 128 / heads), and a single
// decoded token's heads are one tile of the same kernel.
//
//   warp 0     TMA: the Q tile once (one 64-element slice after the other), and the key tiles into a ring;
//              a tile of kKeys keys is row / 64 slices [kKeys][64], each filled page by page
//   warp 1     allocates tensor memory; one lane issues S = Q K^T (row / 16 MMAs, both operands K-major), a
//              tile ahead, and O += P V: P comes from tensor memory, V is the leading slices of the very
//              tile that served as K, read as the MN-major operand
//   warps 2-5  softmax: thread = query row = tensor-memory lane; 32-bit scores, mask, sum; P goes back to tensor
//              memory as bfloat16
//
// Shared memory is what limits the shape: at 576 elements a row the Q tile is 144 KB, so a key tile has 32 keys
// (36 KB) and the ring two stages.  Tensor memory (512 columns) holds two S and two P tiles and an accumulator
// of up to 320 values; longer values are cut over the CTAs of grid z, which each repeat the first product
// (at 512 values: 832 instead of 1,088 multiply-adds per key and row in each of two CTAs).
//
// The accumulator is scaled by a reference m per row: the maximum of the first tile in which the row sees a key,
// moved (with the accumulator) only when a later score exceeds it by 2^16; bfloat16 and 32-bit keep their
// relative precision over that range.  The keys of a few decoded tokens are cut in `splits` (grid z as well),
// whose unnormalised shares latent_decode_merge (attention_generic.cu) adds up; otherwise sink and gate are
// applied here.  Every barrier wait is bounded and reports through the status word.
#include <type_traits>

#include "tcgen05.cuh"

namespace einf {

constexpr int kRows = 128;                  // query rows per CTA = tensor-memory lanes
constexpr int kThreads = 192;
constexpr int kMaxStages = 6;
constexpr int kMaxSlices = 10;              // rows up to 640 elements
constexpr int kMaxValueSlices = 5;          // of the accumulator: 320 of the 512 tensor-memory columns
constexpr int kTmemColumns = 512;
constexpr int kBarBytes = 256;              // q_full, k_full[], k_empty[], s_full[2], p_full[2], o_done[2], the allocation's address
constexpr float kMoveLimit = 16.f;          // exponent of 2 above the reference at which it moves

struct LatentParams {
  const int4* tiles;          // prompt portions: request, first token, tokens (up to 128), first position; or null:
  const int* token_list;      // single tokens by their packed index (null: 0 .. n - 1)
  const int* seq_of_token;
  const int* positions;
  const int* block_table;     // [requests, table_width]
  __nv_bfloat16* out;         // [tokens, heads, value_size]
  float* part_acc;            // [single tokens, heads, splits, value_size], with splits > 1
  float* part_ml;             // [single tokens, heads, splits, 2]: maximum (natural exponent) and sum
  const float* sink;          // see attention_generic.cu
  const float* gate;
  int* status;
  int num_heads, value_size, page_size, num_pages, table_width, window;
  int slices, value_parts, splits, stages, box_keys, q_box_rows;
  float scale_log2;
};

__device__ __forceinline__ void tmem_st8(uint32_t taddr, const uint32_t* v) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"r"(taddr), "r"(v[0]), "r"(v[1]),
               "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7])
               : "memory");
}

// kKeys keys per tile: 16, 32 or 64.
template <int kKeys>
__global__ void __launch_bounds__(kThreads, 1)
latent_attention_tcgen05_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                                const __grid_constant__ LatentParams p) {
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  const uint32_t base = saddr(smem_raw);
  if (base & 1023u) {
    if (threadIdx.x == 0) atomicOr(p.status, kStatusWaitExpired);
    return;
  }
  // --- which rows, which keys, which values ---
  int request, token0, tokens, pos0;
  if (p.tiles) {
    const int4 info = p.tiles[gridDim.x - 1 - blockIdx.x];      // from the last (most keys) to the first
    request = info.x;
    token0 = info.y;
    tokens = info.z;
    pos0 = info.w;
  } else {
    token0 = p.token_list ? p.token_list[blockIdx.x] : (int)blockIdx.x;
    tokens = 1;
    request = p.seq_of_token[token0];
    pos0 = p.positions[token0];
  }
  const int heads = p.num_heads;
  const int row0 = (int)blockIdx.y * kRows;                     // within the tile's tokens * heads rows
  const int rows = min(kRows, tokens * heads - row0);
  if (rows <= 0) return;                                        // the whole CTA: fewer tokens than the grid is made for
  const int part = (int)blockIdx.z % p.value_parts, split = (int)blockIdx.z / p.value_parts;
  const int first_pos = pos0 + row0 / heads, last_pos = pos0 + (row0 + rows - 1) / heads;
  int k_begin = p.window > 0 ? max(0, first_pos - p.window + 1) : 0;
  k_begin = k_begin / p.box_keys * p.box_keys;                  // a TMA box starts on its own multiple
  int k_end = last_pos + 1;
  if (p.splits > 1) {
    const int per = ((k_end - k_begin + kKeys - 1) / kKeys + p.splits - 1) / p.splits * kKeys;
    k_begin = min(k_end, k_begin + split * per);
    k_end = min(k_end, k_begin + per);
  }
  const int num_tiles = (k_end - k_begin + kKeys - 1) / kKeys;
  const int value_slices_all = (p.value_size + 63) / 64;
  const int per_part = (value_slices_all + p.value_parts - 1) / p.value_parts;
  const int v_first = part * per_part, v_slices = min(per_part, value_slices_all - v_first);
  constexpr uint32_t kSlice = kKeys * 128u;                     // a [kKeys x 64] bfloat16 slice of a key tile
  const uint32_t stage_bytes = (uint32_t)p.slices * kSlice;
  const uint32_t q_slice = (uint32_t)p.q_box_rows * 128u;       // a [q_box_rows x 64] bfloat16 slice of Q
  const uint32_t q_addr = base, k_addr = base + (uint32_t)p.slices * q_slice;
  const uint32_t bars = k_addr + (uint32_t)p.stages * stage_bytes;
  const uint32_t q_full = bars;
  auto k_full = [&](int s) { return bars + 8u * (1 + s); };
  auto k_empty = [&](int s) { return bars + 8u * (1 + kMaxStages + s); };
  auto s_full = [&](int b) { return bars + 8u * (1 + 2 * kMaxStages + b); };
  auto p_full = [&](int b) { return bars + 8u * (3 + 2 * kMaxStages + b); };
  auto o_done = [&](int b) { return bars + 8u * (5 + 2 * kMaxStages + b); };   // the second product of an even, an odd tile
  const uint32_t tmem_holder = bars + 8u * (7 + 2 * kMaxStages);
  volatile uint32_t* tmem_holder_ptr = reinterpret_cast<volatile uint32_t*>(smem_raw + (tmem_holder - base));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* table = p.block_table + (size_t)request * p.table_width;

  if (threadIdx.x == 0) {
    bar_init(q_full, 1);
    for (int s = 0; s < kMaxStages; ++s) {
      bar_init(k_full(s), 1);
      bar_init(k_empty(s), 1);
    }
    for (int b = 0; b < 2; ++b) {
      bar_init(s_full(b), 1);
      bar_init(p_full(b), 128);
      bar_init(o_done(b), 1);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tmem_holder), "r"(kTmemColumns)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = *tmem_holder_ptr;
  auto tmem_s = [&](int b) { return tmem + (uint32_t)(kKeys * b); };
  auto tmem_p = [&](int b) { return tmem + (uint32_t)(2 * kKeys + kKeys / 2 * b); };
  const uint32_t tmem_o = tmem + 192u;

  pdl_launch_dependents();   // after the tensor-memory allocation, see gemm_tcgen05.cu
  pdl_wait();
  if (warp == 0) {
    // ---- producer.  Lane j < boxes reads box j's page of a tile, a tile ahead; the requests of a tile (one per box and
    // slice) are spread over the lanes.  A box beyond the last key repeats the last one's page: its keys are
    // masked, but what stands there as values has to be finite. ----
    const int boxes = kKeys / p.box_keys;
    const uint32_t box_bytes = (uint32_t)p.box_keys * 128u;
    if (lane == 0 && num_tiles > 0) bar_expect_tx(q_full, (uint32_t)p.slices * q_slice);
    __syncwarp();
    if (lane < p.slices && num_tiles > 0) tma_2d(q_addr + lane * q_slice, &map_q, lane * 64, token0 * heads + row0, q_full);
    bool bad = false;
    auto row_of_box = [&](int i) {        // cache row at which this lane's box of tile i starts
      if (i >= num_tiles || lane >= boxes) return 0;
      const int key = min(k_begin + i * kKeys + lane * p.box_keys, (k_end - 1) / p.box_keys * p.box_keys);
      const int logical = key / p.page_size;
      int page = table[logical];
      if (page < 0 || page >= p.num_pages) {
        bad = true;
        page = 0;       // keep the byte count right; the status word fails the step
      }
      return page * p.page_size + (key - logical * p.page_size);
    };
    int where = row_of_box(0), issued = 0;
    for (int i = 0; i < num_tiles; ++i, ++issued) {
      const int next = row_of_box(i + 1);
      const int s = i % p.stages;
      if (i >= p.stages && !__all_sync(0xffffffffu, bar_wait(k_empty(s), ((i / p.stages) & 1) ^ 1, p.status))) break;
      if (lane == 0) bar_expect_tx(k_full(s), stage_bytes);
      __syncwarp();
      for (int request0 = 0; request0 < boxes * p.slices; request0 += 32) {
        const int index = request0 + lane;
        const int box = index % boxes, slice = index / boxes;
        const int row = __shfl_sync(0xffffffffu, where, box);
        if (slice < p.slices)
          tma_2d(k_addr + s * stage_bytes + slice * kSlice + box * box_bytes, &map_k, slice * 64, row, k_full(s));
      }
      where = next;
    }
    if (__any_sync(0xffffffffu, bad) && lane == 0) atomicOr(p.status, kStatusBadPage);
    // no copy is in flight when the CTA leaves, whatever went wrong
    if (num_tiles > 0) bar_wait(q_full, 0, p.status);
    for (int i = max(0, issued - p.stages); i < issued; ++i) bar_wait(k_full(i % p.stages), (i / p.stages) & 1, p.status);
  } else if (warp == 1) {
    if (lane == 0 && num_tiles > 0) {
      // ---- both products, the first one a tile ahead of the second ----
      const uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kKeys >> 3) << 17) | ((128u >> 4) << 24);
      const uint64_t desc_q = desc_k_major(q_addr);
      auto first_product = [&](int i) {
        const int s = i % p.stages;
        if (!bar_wait(k_full(s), (i / p.stages) & 1, p.status)) return false;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint64_t desc_k = desc_k_major(k_addr + s * stage_bytes);
        for (int slice = 0; slice < p.slices; ++slice)
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            mma_ss(tmem_s(i & 1), desc_advance(desc_q, slice * q_slice + kk * 32),
                   desc_advance(desc_k, slice * kSlice + kk * 32), idesc_s, (slice > 0 || kk > 0) ? 1u : 0u);
        mma_commit(s_full(i & 1));
        return true;
      };
      bool ok = bar_wait(q_full, 0, p.status) && first_product(0);
      for (int i = 0; i < num_tiles && ok; ++i) {
        // S(i + 1) goes where S(i - 1) stood: that was in registers before P(i - 1) was handed over
        if (i + 1 < num_tiles) ok = first_product(i + 1);
        if (!ok || !(ok = bar_wait(p_full(i & 1), (i >> 1) & 1, p.status))) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const int s = i % p.stages;
        for (int v0 = 0; v0 < v_slices; v0 += 4) {              // up to 256 values an MMA
          const int n = min(4, v_slices - v0) * 64;
          const uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(n >> 3) << 17) | ((128u >> 4) << 24);
          const uint64_t desc_v = desc_mn_major(k_addr + s * stage_bytes + (v_first + v0) * kSlice, kSlice);
#pragma unroll
          for (int ks = 0; ks < kKeys / 16; ++ks)
            mma_ts(tmem_o + v0 * 64, tmem_p(i & 1) + ks * 8, desc_advance(desc_v, ks * 16 * 128), idesc_o,
                   (i > 0 || ks > 0) ? 1u : 0u);
        }
        mma_commit(o_done(i & 1));
        mma_commit(k_empty(s));
      }
    }
  } else {
    // ---- softmax and output: thread r owns query row r ----
    const int r = (warp & 3) * 32 + lane;
    const uint32_t lane_addr = (uint32_t)((warp & 3) * 32) << 16;
    const bool live = r < rows;
    const int token = live ? (row0 + r) / heads : 0, head = live ? (row0 + r) - token * heads : 0;
    const int pos = live ? pos0 + token : -1;
    const int pos_lo = p.window > 0 ? pos - p.window + 1 : 0;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    // The second product of tile i is complete.  Asked now and then only, while the softmax is at tile i + 1 at most:
    // the barrier's phase before (tile i - 2) is long complete, and the one after cannot be.
    auto wait_product = [&](int i) {
      ok = __all_sync(0xffffffffu, bar_wait(o_done(i & 1), (i >> 1) & 1, p.status));
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    };
    for (int i = 0; i < num_tiles; ++i) {
      ok = __all_sync(0xffffffffu, bar_wait(s_full(i & 1), (i >> 1) & 1, p.status));
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      float sv[kKeys];
      if constexpr (kKeys == 16) {
        tmem_ld16(tmem_s(i & 1) + lane_addr, sv);
      } else {
#pragma unroll
        for (int c0 = 0; c0 < kKeys; c0 += 32) tmem_ld32(tmem_s(i & 1) + lane_addr + c0, sv + c0);
      }
      tmem_ld_wait();
      const int key0 = k_begin + i * kKeys;
      const int c_hi = min(pos, k_end - 1) - key0, c_lo = pos_lo - key0;
      const bool masks = !__all_sync(0xffffffffu, c_hi >= kKeys - 1 && c_lo <= 0);
      float top4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < kKeys; ++c) {
        float z = sv[c] * p.scale_log2;
        if (masks) z = (c <= c_hi && c >= c_lo) ? z : -INFINITY;
        sv[c] = z;
        top4[c & 3] = fmaxf(top4[c & 3], z);
      }
      const float top = fmaxf(fmaxf(top4[0], top4[1]), fmaxf(top4[2], top4[3]));
      const bool moves = m == -INFINITY ? top > -INFINITY : top > m + kMoveLimit;
      if (__any_sync(0xffffffffu, moves)) {
        const float to = moves ? top : m;
        const float factor = m == -INFINITY ? 0.f : fast_exp2(m - to);    // nothing seen so far: an accumulator of zeros
        if (i > 0) {
          wait_product(i - 1);
          if (!ok) break;
          for (int c0 = 0; c0 < v_slices * 64; c0 += 32) {
            float v[32];
            tmem_ld32(tmem_o + lane_addr + c0, v);
            tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < 32; ++c) v[c] *= factor;
            tmem_st32(tmem_o + lane_addr + c0, v);
          }
        }
        l *= factor;
        m = to;
      }
      const float shift = m == -INFINITY ? 0.f : m;
      float sum4[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t packed[kKeys / 2];
#pragma unroll
      for (int c = 0; c < kKeys; c += 2) {
        const float a = fast_exp2(sv[c] - shift), b = fast_exp2(sv[c + 1] - shift);
        sum4[c & 3] += a;
        sum4[(c & 3) + 1] += b;
        const __nv_bfloat162 b2 = __floats2bfloat162_rn(a, b);
        packed[c >> 1] = *reinterpret_cast<const uint32_t*>(&b2);
      }
      l += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
      // this P tile's last reader, the second product of tile i - 2, was complete before S(i) was
      if constexpr (kKeys == 16) {
        tmem_st8(tmem_p(i & 1) + lane_addr, packed);
      } else {
#pragma unroll
        for (int c0 = 0; c0 < kKeys / 2; c0 += 16) tmem_st16(tmem_p(i & 1) + lane_addr + c0, packed + c0);
      }
      tmem_st_wait();
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      bar_arrive(p_full(i & 1));
    }
    if (ok && num_tiles > 0) wait_product(num_tiles - 1);
    const size_t row = (size_t)(token0 + token) * heads + head;
    const size_t share = ((size_t)blockIdx.x * heads + head) * p.splits + split;      // of single tokens, in the launch's order
    float factor = 1.f;
    if (p.splits == 1) {
      if (p.sink && m != -INFINITY) l += exp2f(p.sink[head] * 1.4426950408889634f - m);
      factor = l > 0.f ? 1.f / l : 0.f;
      if (p.gate && live) factor *= p.gate[row];
    } else if (live && part == 0) {
      float* ml = p.part_ml + 2 * share;
      ml[0] = m == -INFINITY ? -INFINITY : m * 0.6931471805599453f;
      ml[1] = l;
    }
    const bool vectors = p.value_size % 8 == 0;
    for (int c0 = 0; c0 < v_slices * 64; c0 += 32) {
      float v[32];
      if (ok && num_tiles > 0) {            // uniform over the warp
        tmem_ld32(tmem_o + lane_addr + c0, v);
        tmem_ld_wait();
      } else {
#pragma unroll
        for (int c = 0; c < 32; ++c) v[c] = 0.f;
      }
      const int column = v_first * 64 + c0;
      if (!live) continue;
      if (p.splits > 1) {
        float* o = p.part_acc + share * p.value_size + column;
#pragma unroll
        for (int c = 0; c < 32; ++c)
          if (column + c < p.value_size) o[c] = v[c];
      } else if (vectors) {
        __nv_bfloat16* o = p.out + row * p.value_size + column;
#pragma unroll
        for (int d = 0; d < 32; d += 8) {
          if (column + d >= p.value_size) break;
          uint4 raw;
          __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
          for (int e = 0; e < 4; ++e) h[e] = __floats2bfloat162_rn(v[d + 2 * e] * factor, v[d + 2 * e + 1] * factor);
          *reinterpret_cast<uint4*>(o + d) = raw;
        }
      } else {
        __nv_bfloat16* o = p.out + row * p.value_size + column;
#pragma unroll
        for (int c = 0; c < 32; ++c)
          if (column + c < p.value_size) o[c] = __float2bfloat16_rn(v[c] * factor);
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kTmemColumns) : "memory");
  }
}

struct LatentShape {
  int keys, stages, value_parts, smem;
};

// The key tile of a row size: the largest of which two stages fit beside the Q tile, else one stage of the smallest.
inline LatentShape latent_shape(int slices, int value_size, int q_rows) {
  LatentShape shape = {};
  const int room = 227 * 1024 - slices * q_rows * 128 - kBarBytes;
  for (int keys : {64, 32, 16}) {
    shape.keys = keys;
    shape.stages = room / (slices * keys * 128);
    if (shape.stages >= 2) break;
  }
  if (shape.stages > kMaxStages) shape.stages = kMaxStages;
  const int value_slices = (value_size + 63) / 64;
  shape.value_parts = (value_slices + kMaxValueSlices - 1) / kMaxValueSlices;
  shape.smem = slices * q_rows * 128 + shape.stages * slices * shape.keys * 128 + kBarBytes;
  // one CTA an SM: it takes all of the tensor memory
  if (shape.smem < 116 * 1024) shape.smem = 116 * 1024;
  return shape;
}

}  // namespace einf

using namespace einf;

// CTAs per (128 query rows, split) for values of this size, for the caller's choice of splits.
extern "C" int einf_latent_attention_tcgen05_parts(int value_size) {
  return ((value_size + 63) / 64 + kMaxValueSlices - 1) / kMaxValueSlices;
}

// q: [tokens, heads, row] bfloat16, cache: [pages, 1, page_size, row]; out: [tokens, heads, value_size].  Either `tiles`
// [num_tiles, 4] (prompt portions of up to 128 tokens each) or num_tiles single tokens (token_list, or 0 .. num_tiles - 1;
// then seq_of_token and positions are read).  With splits > 1 the shares go to part_acc and part_ml.
extern "C" int einf_latent_attention_tcgen05(const void* q, const void* cache, const int* block_table, const int* tiles,
                                             const int* token_list, const int* seq_of_token, const int* positions,
                                             int num_tiles, void* out, float* part_acc, float* part_ml, int num_tokens,
                                             int num_heads, int row_size, int value_size, int page_size, int num_pages,
                                             int table_width, float scale, int window, int splits, const float* sink,
                                             const float* gate, int* status, cudaStream_t stream) {
  if (num_tiles == 0) return 0;
  if (row_size % 64 || row_size <= 0 || row_size > 64 * kMaxSlices || value_size <= 0 || value_size > row_size ||
      num_heads <= 0 || page_size < 8 || page_size > 128 || (page_size & (page_size - 1)) || splits < 1 ||
      (splits > 1 && (tiles || !part_acc || !part_ml)) || ((uintptr_t)q & 15) || ((uintptr_t)cache & 15) ||
      ((uintptr_t)out & 15))
    return (int)cudaErrorInvalidValue;
  const int slices = row_size / 64;
  LatentParams p = {};
  p.tiles = (const int4*)tiles;
  p.token_list = token_list;
  p.seq_of_token = seq_of_token;
  p.positions = positions;
  p.block_table = block_table;
  p.out = (__nv_bfloat16*)out;
  p.part_acc = part_acc;
  p.part_ml = part_ml;
  p.sink = sink;
  p.gate = gate;
  p.status = status;
  p.num_heads = num_heads;
  p.value_size = value_size;
  p.page_size = page_size;
  p.num_pages = num_pages;
  p.table_width = table_width;
  p.window = window;
  p.slices = slices;
  p.splits = splits;
  p.scale_log2 = scale * 1.4426950408889634f;
  // Single tokens of a few heads: only their rows of Q are loaded and have a place in shared memory.  The first product
  // still reads 128 rows from there on, the others being whatever stands behind (the key tiles, which are longer):
  // the rows of S that come of it are no one's.
  p.q_box_rows = kRows;
  if (!tiles)
    while (p.q_box_rows / 2 >= num_heads && p.q_box_rows > 8) p.q_box_rows /= 2;
  const LatentShape shape = latent_shape(slices, value_size, p.q_box_rows);
  if (shape.stages < 1) return (int)cudaErrorInvalidValue;
  p.value_parts = shape.value_parts;
  p.stages = shape.stages;
  p.box_keys = page_size < shape.keys ? page_size : shape.keys;
  CUtensorMap map_q, map_k;
  int rc = make_map(&map_q, q, (long long)num_tokens * num_heads, row_size, p.q_box_rows);
  if (rc) return rc;
  rc = make_map(&map_k, cache, (long long)num_pages * page_size, row_size, p.box_keys);
  if (rc) return rc;
  const long long row_tiles = ((tiles ? 128ll : 1ll) * num_heads + kRows - 1) / kRows;
  if (row_tiles > 65535 || (long long)splits * shape.value_parts > 65535) return (int)cudaErrorInvalidValue;
  const dim3 grid(num_tiles, (int)row_tiles, shape.value_parts * splits);
  auto launch = [&](auto kernel) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, shape.smem);
    if (e != cudaSuccess) return (int)e;
    return (int)launch_pdl(kernel, grid, dim3(kThreads), shape.smem, stream, map_q, map_k, p);
  };
  if (shape.keys == 64) return launch(latent_attention_tcgen05_kernel<64>);
  if (shape.keys == 32) return launch(latent_attention_tcgen05_kernel<32>);
  return launch(latent_attention_tcgen05_kernel<16>);
}
