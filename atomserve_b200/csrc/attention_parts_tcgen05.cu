// Paged attention for prompt portions on the fifth-generation tensor cores where a query head holds a
// vector per key head and its score is the sum of their products over all KV key heads (scores mixed
// across heads; see attention_parts.cu, whose prefill kernel serves the shapes this one does not):
// bfloat16, head size 128, causal, with an optional window that may keep the first positions. Both
// products are tcgen05.mma with the scores and the output accumulator in tensor memory, operands by
// TMA (no multicast) straight from the cache pages.
//
// One block per (request, tile of QT query tokens, kv head); its 128 rows are (token, head) pairs.
// Keys are visited in tiles of 128: a tile's scores are one accumulation over KV x 128 entries, so
// Q K^T is several times P V and the block is bound by the first product's operands and issue. Tiles of
// 128 keys (rather than 64) halve the MMAs a score costs their issuing thread.
//
//   warps 0, 8 TMA: the queries of all parts once (where they fit), then the keys in stages of
//              [128 keys][128 entries of one part], the two warps taking turns (a stage's wait,
//              announcement and requests take a warp longer than the MMAs that read it); where the
//              queries do not fit, each stage brings the part's [128 rows][128 entries] of them too.
//   warp 7     TMA: the values, in stages of [64 keys][128 entries].
//   warp 1     MMA: S[b] = sum over parts of Q_c K_c^T into score buffer b = tile & 1.
//   warp 6     MMA: O += P V once the softmax has written P over the scores, where it is the A operand.
//   warps 2-5  softmax: thread r owns row r (a TMEM lane); maxima move lazily (a factor of 256).
//
// Tensor memory: two score buffers of 128 columns and 128 of output, 384 of the 512 allocated (one
// block per SM). All barrier waits are bounded; a wait that runs out sets *status and the roles wind
// down to the final barrier.
#include "tcgen05.cuh"

namespace {

using namespace asb::t5;

constexpr int kThreads = 288;
constexpr int HD = 128;
constexpr int kRows = 128;
constexpr int kKeys = 128;                       // keys per tile
constexpr int kBlockBytes = 128 * 64 * 2;        // [128 rows][64 entries], swizzled: 16 KB
constexpr int kVBlockBytes = 64 * 64 * 2;        // [64 keys][64 entries]: 8 KB
constexpr int kVBytes = 2 * kVBlockBytes;        // a stage of values: 64 keys, both halves of the head
constexpr int kVStages = 2, kMaxKStages = 4;
constexpr int kKBytes = 2 * kBlockBytes;         // a stage of keys (or of queries): 128 rows, both halves of the head
constexpr int kBarrierBytes = 256;
constexpr int kMaxSmem = 227 * 1024;
constexpr uint32_t kTmemCols = 512;
constexpr int kShortRows = 8;

struct PartsParams {
  __nv_bfloat16* out;        // [T, H, HD]
  const int* block_tables;   // [R, table_width]
  const int* req_q_start;    // [R + 1]
  const int* req_pos_start;  // [R]
  int* status;
  int R, H, KV, bs, table_width;
  int G, QT;                 // query heads per kv head, tokens per tile (128 / G)
  int window, keep;          // 0: none
  int k_stages;
  float scale_log2;          // softmax scale times log2(e)
};

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// a ring's next stage and the number of times it has gone round
struct Ring {
  int stage = 0;
  uint32_t round = 0;
  __device__ __forceinline__ void next(int stages) {
    if (++stage == stages) { stage = 0; ++round; }
  }
};

template <bool kStreamQ>
__global__ void __launch_bounds__(kThreads, 1)
parts_prefill_tcgen05_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                             const __grid_constant__ CUtensorMap map_v, const PartsParams p) {
  extern __shared__ __align__(1024) unsigned char smem_raw[];  // the swizzled tiles need this alignment
  const uint32_t base = smem_u32(smem_raw);
  constexpr int kStageBytes = kStreamQ ? 2 * kKBytes : kKBytes;
  const int KS = p.k_stages;
  const uint32_t q_smem = base;  // [KV][2 halves] blocks, where they stay
  const uint32_t k_base = base + (kStreamQ ? 0u : (uint32_t)p.KV * 2u * kBlockBytes);
  auto k_smem = [&](int s) { return k_base + (uint32_t)s * kStageBytes; };
  const uint32_t v_base = k_base + (uint32_t)KS * kStageBytes;
  auto v_smem = [&](int s) { return v_base + (uint32_t)s * kVBytes; };
  const uint32_t bars = v_base + kVStages * kVBytes;
  const uint32_t q_full = bars;
  auto s_full = [&](int b) { return bars + 8u * (1 + b); };
  auto p_full = [&](int b) { return bars + 8u * (3 + b); };
  auto pv_done = [&](int b) { return bars + 8u * (5 + b); };
  auto v_full = [&](int s) { return bars + 8u * (7 + s); };
  auto v_empty = [&](int s) { return bars + 8u * (7 + kVStages + s); };
  auto k_full = [&](int s) { return bars + 8u * (7 + 2 * kVStages + s); };
  auto k_empty = [&](int s) { return bars + 8u * (7 + 2 * kVStages + kMaxKStages + s); };
  constexpr int kBarriers = 7 + 2 * kVStages + 2 * kMaxKStages;
  static_assert(8 * kBarriers + 4 <= kBarrierBytes, "the barriers and the tensor-memory slot");
  volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem_raw + (bars - base) + 8 * kBarriers);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (base & 1023u) {  // the launch did not honour the declared alignment
    if (threadIdx.x == 0) atomicExch(p.status, 19);
    return;
  }

  // Which request and tile of its tokens? (kv head fastest, late tiles first: the longest blocks start first)
  int tile = blockIdx.x / p.KV, r = 0, q_len = 0;
  for (; r < p.R; ++r) {
    q_len = p.req_q_start[r + 1] - p.req_q_start[r];
    if (q_len <= kShortRows) continue;
    const int n = (q_len + p.QT - 1) / p.QT;
    if (tile < n) {
      tile = n - 1 - tile;
      break;
    }
    tile -= n;
  }
  if (r >= p.R) return;  // the whole block leaves before any barrier or allocation
  const int q0 = tile * p.QT, nq = min(p.QT, q_len - q0);
  const int row0 = p.req_q_start[r] + q0, pos0 = p.req_pos_start[r] + q0;
  const int kvh = blockIdx.x % p.KV, head0 = kvh * p.G;
  const int* table = p.block_tables + (size_t)r * p.table_width;
  const int lo = p.window > 0 ? max(0, pos0 - p.window + 1) : 0, hi = pos0 + nq;
  // the kept positions' tiles, then those of the rows' windows
  const int begin = lo / kKeys, kept = min((min(p.keep, lo) + kKeys - 1) / kKeys, begin);
  const int num_tiles = kept + (hi + kKeys - 1) / kKeys - begin;
  auto first_key = [&](int j) { return (j < kept ? j : j - kept + begin) * kKeys; };

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < KS; ++s) {
      mbar_init(k_full(s), 1);
      mbar_init(k_empty(s), 1);
    }
    for (int s = 0; s < kVStages; ++s) {
      mbar_init(v_full(s), 1);
      mbar_init(v_empty(s), 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(s_full(b), 1);
      mbar_init(p_full(b), 4);  // one arrival per softmax warp
      mbar_init(pv_done(b), 1);
    }
    mbar_init_fence();
  }
  if (warp == 1) tmem_alloc(smem_u32((const void*)tmem_slot), kTmemCols);
  fence_before_sync();
  __syncthreads();
  fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;
  auto tmem_s = [&](int j) { return tmem_base + (uint32_t)(j & 1) * kKeys; };
  const uint32_t tmem_o = tmem_base + 2 * kKeys;
  asb::pdl_wait();
  asb::pdl_launch_dependents();

  const int last_page = (hi - 1) / p.bs;
  const uint32_t q_bytes = (uint32_t)(p.QT * p.G * 128);  // a box of queries: QT x G rows, at most 128
  // Pages beyond the request's end, or given back behind the window, are masked out anyway: a page the
  // request holds is read instead, so that shared memory never holds non-finite values.
  auto page_row = [&](int key) {  // row of kv head 0 in the pools
    int blk = table[min(key / p.bs, last_page)];
    if (blk < 0) blk = table[last_page];
    return blk * p.KV * p.bs + key % p.bs;
  };
  if (warp == 0 || warp == 8) {
    if (warp == 0 && lane == 0 && !kStreamQ) {
      mbar_expect_tx(q_full, 2u * p.KV * q_bytes);
      for (int c = 0; c < 2 * p.KV; ++c) tma_load_3d(q_smem + (uint32_t)c * kBlockBytes, &map_q, q_full, c * 64, head0, row0);
    }
    const int box_rows = min(p.bs, kKeys), boxes = kKeys / box_rows;  // rows one box brings; at most 16 boxes of each half
    const int i = lane >> 1, which = lane & 1;                        // a lane's box and half
    const int total = num_tiles * p.KV;
    int row_y = 0, tile_of_row = -1;
    for (int n = warp >> 3; n < total; n += 2) {
      const int j = n / p.KV, c = n - j * p.KV, s = n % KS;
      if (j != tile_of_row && i < boxes) row_y = page_row(first_key(j) + i * box_rows);
      tile_of_row = j;
      int ok_i = 1;
      if (lane == 0) {
        ok_i = mbar_wait(k_empty(s), ((uint32_t)(n / KS) & 1u) ^ 1u, p.status, 11) ? 1 : 0;
        if (ok_i) mbar_expect_tx(k_full(s), (uint32_t)kKBytes + (kStreamQ ? 2u * q_bytes : 0u));
      }
      if (!__shfl_sync(0xffffffffu, ok_i, 0)) break;
      if (i < boxes)
        tma_load_2d(k_smem(s) + (uint32_t)which * kBlockBytes + (uint32_t)(i * box_rows) * 128u, &map_k, k_full(s), which * 64, row_y + c * p.bs);
      if (kStreamQ && lane < 2) tma_load_3d(k_smem(s) + kKBytes + (uint32_t)lane * kBlockBytes, &map_q, k_full(s), c * HD + lane * 64, head0, row0);
    }
  } else if (warp == 7) {
    const int box_rows = min(p.bs, 64), boxes = 64 / box_rows;  // at most 8 boxes of each half
    const int i = lane >> 1, which = lane & 1;
    for (int n = 0; n < 2 * num_tiles; ++n) {
      const int s = n % kVStages;
      const int row_y = i < boxes ? page_row(first_key(n >> 1) + (n & 1) * 64 + i * box_rows) + kvh * p.bs : 0;
      int ok_i = 1;
      if (lane == 0) {
        ok_i = mbar_wait(v_empty(s), ((uint32_t)(n / kVStages) & 1u) ^ 1u, p.status, 21) ? 1 : 0;
        if (ok_i) mbar_expect_tx(v_full(s), (uint32_t)kVBytes);
      }
      if (!__shfl_sync(0xffffffffu, ok_i, 0)) break;
      if (i < boxes) tma_load_2d(v_smem(s) + (uint32_t)which * kVBlockBytes + (uint32_t)(i * box_rows) * 128u, &map_v, v_full(s), which * 64, row_y);
    }
  } else if (warp == 1) {
    // S = Q K^T, a tile ahead of the softmax
    if (lane == 0) {
      constexpr uint32_t idesc_qk = instr_desc_bf16(kRows, kKeys, false);
      bool ok = kStreamQ || mbar_wait(q_full, 0, p.status, 12);
      const int total = num_tiles * p.KV;
      Ring ring;
      for (int n = 0, j = 0, c = 0; n < total && ok; ++n) {
        // score buffer j & 1 held tile j - 2's scores and then its P: has that tile's P V read it?
        if (c == 0 && j >= 2) ok = mbar_wait(pv_done(j & 1), ((uint32_t)(j - 2) >> 1) & 1u, p.status, 18);
        const int s = ring.stage;
        if (ok) ok = mbar_wait(k_full(s), ring.round & 1u, p.status, 13);
        if (!ok) break;
        fence_after_sync();
        ring.next(KS);
        const uint32_t q_block = kStreamQ ? k_smem(s) + kKBytes : q_smem + (uint32_t)c * kKBytes;
#pragma unroll
        for (int ks = 0; ks < HD / 16; ++ks) {  // 16 entries per MMA: 32 bytes along the swizzled row
          const uint32_t at = (uint32_t)(ks / 4) * kBlockBytes + (uint32_t)(ks % 4) * 32u;
          umma_bf16(tmem_s(j), desc_k_major(q_block + at, 1024), desc_k_major(k_smem(s) + at, 1024), idesc_qk, (uint32_t)((c | ks) != 0));
        }
        umma_commit(k_empty(s));
        if (++c == p.KV) {
          umma_commit(s_full(j & 1));
          c = 0;
          ++j;
        }
      }
    }
  } else if (warp == 6) {
    // O += P V as soon as the softmax has written a tile's P
    if (lane == 0) {
      constexpr uint32_t idesc_pv = instr_desc_bf16(kRows, HD, true);
      bool ok = true;
      Ring ring;
      for (int j = 0; j < num_tiles && ok; ++j) {
        ok = mbar_wait(p_full(j & 1), ((uint32_t)j >> 1) & 1u, p.status, 15);
        for (int sub = 0; sub < 2 && ok; ++sub) {
          const int s = ring.stage;
          ok = mbar_wait(v_full(s), ring.round & 1u, p.status, 22);
          if (!ok) break;
          fence_after_sync();
#pragma unroll
          for (int ks = 0; ks < 4; ++ks) {  // 16 keys per MMA: eight 32-bit columns of P
            const uint64_t b = desc_mn_major(v_smem(s) + (uint32_t)ks * 2048u, kVBlockBytes, 1024);
            umma_bf16_a_tmem(tmem_o, tmem_s(j) + (uint32_t)(sub * 4 + ks) * 8u, b, idesc_pv, (uint32_t)((j | sub | ks) != 0));
          }
          umma_commit(v_empty(s));
          ring.next(kVStages);
        }
        if (ok) umma_commit(pv_done(j & 1));
      }
    }
  } else {
    // Softmax and epilogue: thread `row` of the block owns TMEM lane `row`.
    const int quad = warp & 3, row = quad * 32 + lane, qi = row / p.G;
    const bool real = qi < nq;
    const int pos = real ? pos0 + qi : -1;  // padding rows see nothing
    const int row_lo = p.window > 0 ? pos - p.window + 1 : 0;
    const uint32_t lane_addr = (uint32_t)(quad * 32) << 16;
    const bool real_block = nq * p.G == kRows;
    const float mul = p.scale_log2;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    uint32_t scores_there = 0;  // lane 0: the answer to an early question about this tile's scores
    for (int j = 0; j < num_tiles && ok; ++j) {
      const int kt0 = first_key(j);
      int ok_i = 1;
      if (lane == 0 && !scores_there) ok_i = mbar_wait(s_full(j & 1), ((uint32_t)j >> 1) & 1u, p.status, 16) ? 1 : 0;
      ok = __shfl_sync(0xffffffffu, ok_i, 0) != 0;
      if (!ok) break;
      fence_after_sync();
      // tiles strictly inside every row's view need no mask
      const bool inside = kt0 + kKeys <= pos0 + 1 && real_block && (p.window <= 0 || kt0 > hi - 1 - p.window || kt0 + kKeys <= p.keep);
      uint32_t raw[kKeys];
#pragma unroll
      for (int c = 0; c < kKeys; c += 32) tmem_ld32_nowait(tmem_s(j) + lane_addr + (uint32_t)c, raw + c);
      tmem_ld_wait();
      float part_max[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) part_max[u] = -INFINITY;
      if (!inside) {
#pragma unroll
        for (int i = 0; i < kKeys; ++i) {
          const int key = kt0 + i;
          if (!(key <= pos && (key >= row_lo || key < p.keep))) raw[i] = 0xff800000u;  // -inf
        }
      }
#pragma unroll
      for (int i = 0; i < kKeys; ++i) part_max[i & 7] = fmaxf(part_max[i & 7], __uint_as_float(raw[i]));
      const float raw_max = fmaxf(fmaxf(fmaxf(part_max[0], part_max[1]), fmaxf(part_max[2], part_max[3])),
                                  fmaxf(fmaxf(part_max[4], part_max[5]), fmaxf(part_max[6], part_max[7])));
      const float tile_max = raw_max * mul;  // the scale is positive
      // the running maximum moves only when the new one exceeds it by more than 8 (log2 units)
      float corr = 1.f;
      if (tile_max > m + 8.f || (m == -INFINITY && tile_max > -INFINITY)) {
        const float m_new = fmaxf(m, tile_max);
        corr = fast_exp2(m - m_new);  // 0 when m was -inf
        m = m_new;
        l *= corr;
      }
      const float m_use = m == -INFINITY ? 0.f : m;
      if (lane == 0) scores_there = j + 1 < num_tiles ? mbar_try(s_full((j + 1) & 1), ((uint32_t)(j + 1) >> 1) & 1u) : 0u;
      if (j > 0 && __any_sync(0xffffffffu, corr != 1.f)) {
        // rescale this row of O: the previous P V must have completed
        if (lane == 0) ok_i = mbar_wait(pv_done((j - 1) & 1), ((uint32_t)(j - 1) >> 1) & 1u, p.status, 17) ? 1 : 0;
        ok = __shfl_sync(0xffffffffu, ok_i, 0) != 0;
        if (!ok) break;
        fence_after_sync();
#pragma unroll 1
        for (int c = 0; c < HD; c += 32) {
          uint32_t oraw[32];
          tmem_ld32(tmem_o + lane_addr + (uint32_t)c, oraw);
#pragma unroll
          for (int i = 0; i < 32; ++i) oraw[i] = __float_as_uint(__uint_as_float(oraw[i]) * corr);
          tmem_st32(tmem_o + lane_addr + (uint32_t)c, oraw);
        }
        tmem_st_wait();
      }
      // probabilities, their sum, and P as bfloat16 over the first half of the tile's score columns
      const float neg_m = -m_use;
      float part_sum[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t packed[32];
#pragma unroll
        for (int i = 0; i < 64; i += 2) {
          const float a = fast_exp2(fmaf(__uint_as_float(raw[c * 64 + i]), mul, neg_m));
          const float b = fast_exp2(fmaf(__uint_as_float(raw[c * 64 + i + 1]), mul, neg_m));
          part_sum[(i >> 1) & 3] += a + b;
          __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
          packed[i >> 1] = *reinterpret_cast<uint32_t*>(&v);
        }
        tmem_st32(tmem_s(j) + lane_addr + (uint32_t)c * 32u, packed);
      }
      l += (part_sum[0] + part_sum[1]) + (part_sum[2] + part_sum[3]);
      tmem_st_wait();
      fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full(j & 1));
    }
    // epilogue: O / sum, rounded once
    if (ok) {
      int ok_i = 1;
      if (lane == 0) ok_i = mbar_wait(pv_done((num_tiles - 1) & 1), ((uint32_t)(num_tiles - 1) >> 1) & 1u, p.status, 23) ? 1 : 0;
      ok = __shfl_sync(0xffffffffu, ok_i, 0) != 0;
    }
    if (ok) {
      fence_after_sync();
      const float inv = real ? 1.f / l : 0.f;
      __nv_bfloat16* o = p.out + ((size_t)(row0 + qi) * p.H + head0 + (row - qi * p.G)) * HD;
#pragma unroll 1
      for (int c = 0; c < HD; c += 32) {
        uint32_t raw[32];
        tmem_ld32(tmem_o + lane_addr + (uint32_t)c, raw);
        if (real) {
          uint4 v[4];
          __nv_bfloat162* h2 = reinterpret_cast<__nv_bfloat162*>(v);
#pragma unroll
          for (int i = 0; i < 32; i += 2)
            h2[i >> 1] = __floats2bfloat162_rn(__uint_as_float(raw[i]) * inv, __uint_as_float(raw[i + 1]) * inv);
#pragma unroll
          for (int q4 = 0; q4 < 4; ++q4) *reinterpret_cast<uint4*>(o + c + q4 * 8) = v[q4];
        }
      }
    }
  }

  fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    fence_after_sync();
    tmem_dealloc(tmem_base, kTmemCols);
  }
}

// stages of keys that fit beside the queries of all parts; 0: too few, the queries travel with the keys
int resident_stages(int KV) {
  const int left = kMaxSmem - KV * kKBytes - kVStages * kVBytes - kBarrierBytes;
  const int stages = left > 0 ? left / kKBytes : 0;
  return stages >= 2 ? (stages < kMaxKStages ? stages : kMaxKStages) : 0;
}

}  // namespace

// 1 if this kernel serves the shape: head size 128, 1 to 64 query heads per kv head, pages of 8 to 256
// tokens (a power of two).
extern "C" int asb_attention_parts_tcgen05_supported(int hd, int group, int block_size) {
  const bool pow2_page = block_size >= 8 && block_size <= 256 && (block_size & (block_size - 1)) == 0;
  return hd == HD && group >= 1 && group <= 64 && pow2_page ? 1 : 0;
}

// Attention for every request that brings more than 8 tokens (others are left untouched). q
// [T, H, KV, 128], out [T, H, 128] bfloat16; caches [num_blocks, KV, bs, 128].
extern "C" int asb_attention_parts_tcgen05(void* out, const void* q, const void* k_cache, const void* v_cache,
                                           const int* block_tables, const int* req_q_start, const int* req_pos_start,
                                           int num_tokens, int R, int H, int KV, int hd, int bs, int num_blocks,
                                           int table_width, int window, int keep, float scale, int* status,
                                           cudaStream_t stream) {
  if (num_tokens == 0 || R == 0) return 0;
  if (KV < 1 || H % KV) return asb::fail("attention_parts_tcgen05: %d heads over %d kv heads", H, KV);
  if (!asb_attention_parts_tcgen05_supported(hd, H / KV, bs))
    return asb::fail("attention_parts_tcgen05: head_dim %d, group %d, page %d are not served", hd, H / KV, bs);
  if (!status) return asb::fail("attention_parts_tcgen05: a status word is required");
  if (window < 0 || keep < 0 || !(scale > 0.f)) return asb::fail("attention_parts_tcgen05: window %d, keep %d, scale %f", window, keep, (double)scale);
  PartsParams p;
  p.out = (__nv_bfloat16*)out;
  p.block_tables = block_tables; p.req_q_start = req_q_start; p.req_pos_start = req_pos_start; p.status = status;
  p.R = R; p.H = H; p.KV = KV; p.bs = bs; p.table_width = table_width;
  p.G = H / KV;
  p.QT = kRows / p.G;
  p.window = window; p.keep = window > 0 ? keep : 0;
  p.scale_log2 = scale * 1.4426950408889634f;
  const int stages = resident_stages(KV);
  p.k_stages = stages ? stages : 3;
  const int smem = (stages ? (KV + stages) * kKBytes : p.k_stages * 2 * kKBytes) + kVStages * kVBytes + kBarrierBytes;

  alignas(64) CUtensorMap mq, mk, mv;
  {
    const cuuint64_t dims[3] = {(cuuint64_t)KV * HD, (cuuint64_t)H, (cuuint64_t)num_tokens};
    const cuuint64_t strides[2] = {(cuuint64_t)KV * HD * 2, (cuuint64_t)H * KV * HD * 2};
    const cuuint32_t box[3] = {64, (cuuint32_t)p.G, (cuuint32_t)p.QT};
    if (int rc = make_bf16_map(&mq, q, 3, dims, strides, box)) return rc;
  }
  {
    const cuuint64_t dims[2] = {(cuuint64_t)HD, (cuuint64_t)num_blocks * KV * bs};
    const cuuint64_t strides[1] = {(cuuint64_t)HD * 2};
    const cuuint32_t box_k[2] = {64, (cuuint32_t)(bs < kKeys ? bs : kKeys)}, box_v[2] = {64, (cuuint32_t)(bs < 64 ? bs : 64)};
    if (int rc = make_bf16_map(&mk, k_cache, 2, dims, strides, box_k)) return rc;
    if (int rc = make_bf16_map(&mv, v_cache, 2, dims, strides, box_v)) return rc;
  }
  const long long blocks = (long long)((num_tokens + p.QT - 1) / p.QT + R) * KV;
  if (blocks > 0x7fffffffLL) return asb::fail("attention_parts_tcgen05: %lld blocks exceed the grid", blocks);
  auto start = [&](auto kern) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return asb::fail("attention_parts_tcgen05: shared memory %d: %s", smem, cudaGetErrorString(e));
    asb::launch(kern, dim3((unsigned)blocks), kThreads, (size_t)smem, stream, mq, mk, mv, p);
    return asb::check_launch("attention_parts_tcgen05");
  };
  return stages ? start(parts_prefill_tcgen05_kernel<false>) : start(parts_prefill_tcgen05_kernel<true>);
}
