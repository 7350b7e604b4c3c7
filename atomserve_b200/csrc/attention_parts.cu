// Paged attention for bfloat16 on the tensor cores (mma.sync) where a query head holds a vector per
// key head and its score is the sum of their products, score_h = sum_c q[h, c] . k_c over all KV key
// heads (scores mixed across heads: the mix is part of the queries, mixed_heads.cu); its values are
// those of its own kv head h / G. Head sizes 64 and 128, any number of heads and kv heads, causal, with
// an optional sliding window that may keep the sequence's first positions visible. Two kernels:
//
//   decode   one block per (new token, up to 32 query heads, key partition): the heads are the rows
//            of one or two 16-row tiles, so a key is read once for all of them. Per tile of 64 keys the block
//            walks the KV key heads, the scores growing in registers, and then the value heads that
//            its rows belong to, each with the other rows' weights at zero. Four warps per row tile
//            share the keys, sixteen apiece, and merge at the end. Serves requests of at most kShortRows tokens.
//   prefill  one block per (request, tile of tokens, kv head): 128 rows = (token, head) pairs, sixteen
//            per warp; per tile of 64 keys the KV key heads, then the kv head's values. The queries
//            of all parts stay in shared memory where they fit; otherwise a part's queries come with
//            its keys. Serves the longer portions (head size 128 with few parts:
//            attention_parts_tcgen05.cu).
//
// Keys and values travel as items of one ring of shared-memory stages, so that an item's copy is in
// flight while the items before it are multiplied. The tiles a row needs are the kept ones and those
// of its window; partitions cut this list, not the positions in between. Scores, maxima, sums and the
// accumulator are float32; probabilities are rounded to bfloat16 only as the operand of the second
// product, the output once.
#include "attention_mma.cuh"

namespace {

using namespace asb::mma;

constexpr int kKeyTile = 64;
constexpr int kShortRows = 8;  // requests with at most this many new tokens go row by row
constexpr int kPrefillThreads = 256, kPrefillRows = 128;

struct PartsParams {
  const __nv_bfloat16* q;        // [T, H, KV, HD]
  __nv_bfloat16* out;            // [T, H, HD]
  const __nv_bfloat16* k_cache;  // [num_blocks, KV, bs, HD]
  const __nv_bfloat16* v_cache;
  const int* block_tables;       // [R, table_width]
  const int* req_q_start;        // [R + 1]
  const int* req_pos_start;      // [R]
  float* part_m;                 // [rows, H, NP]
  float* part_l;
  float* part_acc;               // [rows, H, NP, HD]
  int T, R, H, KV, bs, table_width;
  int G;                         // query heads per kv head
  int GC, HC;                    // decode: heads per block (<= 32) and blocks; prefill: the same within a kv head
  int QT;                        // prefill: tokens per 128-row tile
  int window, keep;              // 0: none
  int PT, NP;                    // key tiles per partition, partitions (decode)
  int all_single, short_rows;    // as in attention_mma.cu
  float scale;
};

// The tiles of 64 keys that rows see whose first key behind the kept ones is `lo` and whose last is
// `hi` - 1: the kept positions' tiles before the window's, then the window's.
struct TileList {
  int kept, begin, count;
  __device__ __forceinline__ TileList(int lo, int hi, int keep) {
    begin = lo / kKeyTile;
    kept = min((min(keep, lo) + kKeyTile - 1) / kKeyTile, begin);
    count = kept + (hi + kKeyTile - 1) / kKeyTile - begin;
  }
  __device__ __forceinline__ int first_key(int t) const { return (t < kept ? t : t - kept + begin) * kKeyTile; }
};

// How a thread copies a tile of 64 keys (or values) of one kv head: one 16-byte column of a run of
// consecutive positions. Where the run lies inside one page, the page is looked up once per tile, and
// for the next tile while this one's heads are copied.
template <int HD, int NT>
struct TileCopy {
  static constexpr int kChunks = HD / 8, kRun = kKeyTile / (NT / kChunks);
  int chunk, run0, ahead = 0, block = 0;
  bool one_page;

  __device__ __forceinline__ TileCopy(const PartsParams& p)
      : chunk(threadIdx.x % kChunks), run0(threadIdx.x / kChunks * kRun), one_page(p.bs >= kRun && (p.bs & (p.bs - 1)) == 0) {}

  // ask for the page of the thread's run in the tile at kt0 (the answer is taken up by `enter`)
  __device__ __forceinline__ void look(const PartsParams& p, const int* table, int kt0, int lo, int hi, int keep) {
    const int j0 = kt0 + run0;
    if (one_page && j0 < hi && (j0 + kRun > lo || j0 < keep)) ahead = table[j0 / p.bs];
  }
  __device__ __forceinline__ void enter() { block = ahead; }

  // positions that no row sees are zero
  __device__ __forceinline__ void load(uint32_t tile, const __nv_bfloat16* cache, const PartsParams& p, const int* table, int head,
                                       int kt0, int lo, int hi, int keep) const {
    const int j0 = kt0 + run0;
    const size_t page_at = (((size_t)block * p.KV + head) * p.bs + (j0 & (p.bs - 1))) * HD + chunk * 8;
#pragma unroll
    for (int i = 0; i < kRun; ++i) {
      const int j = j0 + i;
      const bool valid = j < hi && (j >= lo || j < keep);
      size_t at = 0;
      if (valid) at = one_page ? page_at + (size_t)i * HD : (((size_t)table[j / p.bs] * p.KV + head) * p.bs + j % p.bs) * HD + chunk * 8;
      cp_async16(tile + tile_offset<HD>(run0 + i, chunk), cache + at, valid);
    }
  }
};

// ---- decode ------------------------------------------------------------------------------------

// WG: groups of four warps, each with 16 query heads of its own and all of a tile's keys; NS: stages of
// the ring (with four, two blocks share an SM)
template <int HD, int WG, int NS>
__global__ void __launch_bounds__(128 * WG, NS == 4 ? 2 : 1)
parts_decode_kernel(const PartsParams p) {
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  extern __shared__ __align__(128) unsigned char smem_raw[];
  constexpr int kTileBytes = kKeyTile * HD * 2, kThreads = 128 * WG, kRows = 16 * WG, kQPart = kRows * HD * 2;
  const uint32_t smem = smem_u32(smem_raw);
  auto stage = [&](int n) { return smem + (uint32_t)(n % NS) * kTileBytes; };
  const uint32_t q_tile = smem + NS * kTileBytes;  // [KV][kRows]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int row = blockIdx.x, r;
  if (p.all_single) {
    r = row;
  } else if (p.short_rows > 0) {
    row = asb::nth_short_row(p.req_q_start, p.R, kShortRows, blockIdx.x, &r);
    if (row < 0) return;
  } else {
    r = find_request(p.req_q_start, p.R, row);
    if (p.req_q_start[r + 1] - p.req_q_start[r] > kShortRows) return;  // the prefill kernel's
  }
  const int pos = p.req_pos_start[r] + (row - p.req_q_start[r]);
  const int head0 = blockIdx.y * p.GC, gc = min(p.GC, p.H - head0);
  const int c_lo = head0 / p.G, values = (head0 + gc - 1) / p.G - c_lo + 1;  // the value heads of these rows
  const int items = p.KV + values;                                          // per tile
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int* table = p.block_tables + (size_t)r * p.table_width;
  const TileList tiles(lo, pos + 1, p.keep);
  const int t_begin = blockIdx.z * p.PT, t_end = min(tiles.count, t_begin + p.PT);
  const int total = max(0, t_end - t_begin) * items;

  TileCopy<HD, kThreads> copy(p);
  int load_kt0 = tiles.first_key(t_begin), next_kt0 = 0, load_tile_no = t_begin, load_item = 0, loaded = 0;
  if (total > 0) copy.look(p, table, load_kt0, lo, pos + 1, p.keep);
  auto load_next = [&]() {
    if (loaded < total) {
      if (load_item == 0) {
        if (load_tile_no > t_begin) load_kt0 = next_kt0;
        copy.enter();
        if (++load_tile_no < t_end) {
          next_kt0 = tiles.first_key(load_tile_no);
          copy.look(p, table, next_kt0, lo, pos + 1, p.keep);
        }
      }
      const bool key = load_item < p.KV;
      copy.load(stage(loaded), key ? p.k_cache : p.v_cache, p, table, key ? load_item : c_lo + load_item - p.KV, load_kt0, lo, pos + 1, p.keep);
      if (++load_item == items) load_item = 0;
      ++loaded;
    }
    cp_async_commit();
  };
  for (int n = 0; n < NS - 1; ++n) load_next();
  {  // queries: gc heads of this token, part by part; zero rows above gc
    constexpr int kChunks = HD / 8;
    for (int i = threadIdx.x; i < p.KV * kRows * kChunks; i += kThreads) {
      const int c = i / (kRows * kChunks), qr = i / kChunks % kRows, ch = i % kChunks;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (qr < gc) v = *reinterpret_cast<const uint4*>(p.q + (((size_t)row * p.H + head0 + qr) * p.KV + c) * HD + ch * 8);
      *reinterpret_cast<uint4*>(smem_raw + (q_tile - smem) + c * kQPart + tile_offset<HD>(qr, ch)) = v;
    }
  }

  float m[2], l[2], acc[HD / 8][4], s[2][4];
  uint32_t pf[4] = {0, 0, 0, 0};
  const int group = warp >> 2;         // this warp's 16 heads
  const int key0 = (warp & 3) * 16;    // and its keys inside a tile
  int owner[2];                        // the value heads of a thread's two rows
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    m[h] = -INFINITY;
    l[h] = 0.f;
    owner[h] = (head0 + group * 16 + (lane >> 2) + h * 8) / p.G;
  }
#pragma unroll
  for (int i = 0; i < HD / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  const int krow = key0 + (lane & 7) + ((lane >> 4) << 3), kchunk = (lane >> 3) & 1;
  const int qrow = group * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), qchunk = lane >> 4;

  int item = 0, kt0 = 0, tile = t_begin;
  bool live = false;
  for (int n = 0; n < total; ++n) {
    cp_async_wait<NS - 2>();
    __syncthreads();  // item n has landed; everybody is done with the stage that the next load takes
    load_next();
    if (item == 0) {
      kt0 = tiles.first_key(tile);
      const int first = kt0 + key0;
      live = first <= pos && (first + 16 > lo || first < p.keep);  // uniform in the warp
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
    }
    if (live) {
      if (item < p.KV) {
        const uint32_t q_part = q_tile + (uint32_t)item * kQPart, k_tile = stage(n);
#pragma unroll
        for (int kc = 0; kc < HD / 16; ++kc) {
          uint32_t a[4], b[4];
          ldmatrix_x4(a, q_part + tile_offset<HD>(qrow, kc * 2 + qchunk));
          ldmatrix_x4(b, k_tile + tile_offset<HD>(krow, kc * 2 + kchunk));
          mma_bf16(s[0], a, b[0], b[1]);
          mma_bf16(s[1], a, b[2], b[3]);
        }
        if (item == p.KV - 1) {
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int key = kt0 + key0 + j * 8 + (lane & 3) * 2 + (e & 1);
              s[j][e] = key <= pos && (key >= lo || key < p.keep) ? s[j][e] * p.scale : -INFINITY;
            }
          float rmax[2] = {fmaxf(fmaxf(s[0][0], s[0][1]), fmaxf(s[1][0], s[1][1])),
                           fmaxf(fmaxf(s[0][2], s[0][3]), fmaxf(s[1][2], s[1][3]))};
          float corr[2], rsum[2] = {0.f, 0.f};
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            rmax[h] = fmaxf(rmax[h], __shfl_xor_sync(0xffffffffu, rmax[h], 1));
            rmax[h] = fmaxf(rmax[h], __shfl_xor_sync(0xffffffffu, rmax[h], 2));
            const float m_new = fmaxf(m[h], rmax[h]);  // finite: a live warp sees at least one of its keys
            corr[h] = __expf(m[h] - m_new);
            m[h] = m_new;
          }
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              s[j][e] = __expf(s[j][e] - m[e >> 1]);
              rsum[e >> 1] += s[j][e];
            }
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            rsum[h] += __shfl_xor_sync(0xffffffffu, rsum[h], 1);
            rsum[h] += __shfl_xor_sync(0xffffffffu, rsum[h], 2);
            l[h] = l[h] * corr[h] + rsum[h];
          }
#pragma unroll
          for (int i = 0; i < HD / 8; ++i) {
            acc[i][0] *= corr[0]; acc[i][1] *= corr[0];
            acc[i][2] *= corr[1]; acc[i][3] *= corr[1];
          }
          pf[0] = pack_bf16(s[0][0], s[0][1]); pf[1] = pack_bf16(s[0][2], s[0][3]);
          pf[2] = pack_bf16(s[1][0], s[1][1]); pf[3] = pack_bf16(s[1][2], s[1][3]);
        }
      } else {
        const int c = c_lo + item - p.KV;  // rows of other value heads weigh nothing here
        const uint32_t own[4] = {owner[0] == c ? pf[0] : 0u, owner[1] == c ? pf[1] : 0u, owner[0] == c ? pf[2] : 0u,
                                 owner[1] == c ? pf[3] : 0u};
        const int first_row = c * p.G - head0 - group * 16;
        if (first_row < 16 && first_row + p.G > 0) pv_16keys<HD>(acc, own, stage(n), key0, lane);  // (else none of this group's rows)
      }
    }
    if (++item == items) { item = 0; ++tile; }
  }
  cp_async_wait<0>();
  __syncthreads();

  // Merge the four warps through shared memory (over the stages): per row max, sum, acc.
  float* mm = reinterpret_cast<float*>(smem_raw);  // [4][kRows]
  float* ml = mm + 4 * kRows;                      // [4][kRows]
  float* ma = ml + 4 * kRows;                      // [4][kRows][HD]
  {
    const int g = lane >> 2, q = lane & 3;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int rr = group * 16 + h * 8 + g, at = (warp & 3) * kRows + rr;
      if (q == 0) {
        mm[at] = m[h];
        ml[at] = l[h];
      }
      if (rr < gc) {
#pragma unroll
        for (int i = 0; i < HD / 8; ++i)
          *reinterpret_cast<float2*>(ma + (size_t)at * HD + i * 8 + q * 2) = make_float2(acc[i][2 * h], acc[i][2 * h + 1]);
      }
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < gc * HD; i += kThreads) {
    const int qr = i / HD, col = i - qr * HD;
    float mx = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w)
      if (ml[w * kRows + qr] > 0.f) mx = fmaxf(mx, mm[w * kRows + qr]);
    float a = 0.f, den = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w)
      if (ml[w * kRows + qr] > 0.f) {
        const float f = __expf(mm[w * kRows + qr] - mx);
        den += ml[w * kRows + qr] * f;
        a += ma[(size_t)(w * kRows + qr) * HD + col] * f;
      }
    if (p.NP == 1) {
      p.out[((size_t)row * p.H + head0 + qr) * HD + col] = __float2bfloat16_rn(a / den);
    } else {
      const size_t at = ((size_t)(p.short_rows > 0 ? blockIdx.x : row) * p.H + head0 + qr) * p.NP + blockIdx.z;
      p.part_acc[at * HD + col] = a;
      if (col == 0) {
        p.part_m[at] = mx;
        p.part_l[at] = den;
      }
    }
  }
}

// ---- prefill -----------------------------------------------------------------------------------

constexpr int kPrefillStages = 3;

template <int HD, bool kStreamQ>
__global__ void __launch_bounds__(kPrefillThreads)
parts_prefill_kernel(const PartsParams p) {
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  extern __shared__ __align__(128) unsigned char smem_raw[];
  constexpr int kTileBytes = kKeyTile * HD * 2, kQPart = kPrefillRows * HD * 2;
  constexpr int kStageBytes = kTileBytes + (kStreamQ ? kQPart : 0);
  const uint32_t smem = smem_u32(smem_raw);
  auto stage = [&](int n) { return smem + (uint32_t)(n % kPrefillStages) * kStageBytes; };
  const uint32_t q_all = smem + kPrefillStages * kStageBytes;  // [KV][128 rows] where they stay

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int chunks = p.KV * p.HC, chunk = blockIdx.x % chunks;
  int qtile = blockIdx.x / chunks, r = 0, q_len = 0;
  for (; r < p.R; ++r) {
    q_len = p.req_q_start[r + 1] - p.req_q_start[r];
    if (q_len <= kShortRows) continue;
    const int n = (q_len + p.QT - 1) / p.QT;
    if (qtile < n) {
      qtile = n - 1 - qtile;  // late tiles see the most keys: start them first
      break;
    }
    qtile -= n;
  }
  if (r >= p.R) return;
  const int q0 = qtile * p.QT, nq = min(p.QT, q_len - q0);
  const int row0 = p.req_q_start[r] + q0, pos0 = p.req_pos_start[r] + q0;
  const int kvh = chunk / p.HC, head0 = kvh * p.G + (chunk % p.HC) * p.GC, gc = min(p.GC, kvh * p.G + p.G - head0);
  const int num_rows = nq * gc;  // tile row rr = qi * gc + g
  const int* table = p.block_tables + (size_t)r * p.table_width;
  const int lo = p.window > 0 ? max(0, pos0 - p.window + 1) : 0, hi = pos0 + nq;
  const TileList tiles(lo, hi, p.keep);
  const int items = p.KV + 1, total = tiles.count * items;

  auto load_queries = [&](uint32_t at, int c) {
    constexpr int kChunks = HD / 8;
    for (int i = threadIdx.x; i < kPrefillRows * kChunks; i += kPrefillThreads) {
      const int rr = i / kChunks, ch = i % kChunks;
      const bool real = rr < num_rows;
      const int qi = real ? rr / gc : 0, g = real ? rr - qi * gc : 0;
      cp_async16(at + tile_offset<HD>(rr, ch), p.q + (((size_t)(row0 + qi) * p.H + head0 + g) * p.KV + c) * HD + ch * 8, real);
    }
  };
  TileCopy<HD, kPrefillThreads> copy(p);
  int load_kt0 = tiles.first_key(0), next_kt0 = 0, load_tile_no = 0, load_item = 0, loaded = 0;
  copy.look(p, table, load_kt0, lo, hi, p.keep);
  auto load_next = [&]() {
    if (loaded < total) {
      if (load_item == 0) {
        if (load_tile_no > 0) load_kt0 = next_kt0;
        copy.enter();
        if (++load_tile_no < tiles.count) {
          next_kt0 = tiles.first_key(load_tile_no);
          copy.look(p, table, next_kt0, lo, hi, p.keep);
        }
      }
      const bool key = load_item < p.KV;
      copy.load(stage(loaded), key ? p.k_cache : p.v_cache, p, table, key ? load_item : kvh, load_kt0, lo, hi, p.keep);
      if (kStreamQ && key) load_queries(stage(loaded) + kTileBytes, load_item);
      if (++load_item == items) load_item = 0;
      ++loaded;
    }
    cp_async_commit();
  };
  if (!kStreamQ)
    for (int c = 0; c < p.KV; ++c) load_queries(q_all + (uint32_t)c * kQPart, c);  // (complete with the first item's group)
  for (int n = 0; n < kPrefillStages - 1; ++n) load_next();

  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float acc[HD / 8][4];
#pragma unroll
  for (int i = 0; i < HD / 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  float s[kKeyTile / 8][4];

  int qpos[2];  // positions of this thread's two rows; -1: a padding row, sees nothing
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int rr = warp * 16 + (lane >> 2) + h * 8;
    qpos[h] = rr < num_rows ? pos0 + rr / gc : -1;
  }
  const int warp_first = warp * 16, warp_last = min(warp * 16 + 15, num_rows - 1);
  const int warp_min_pos = pos0 + warp_first / gc, warp_max_pos = warp_first < num_rows ? pos0 + warp_last / gc : -1;
  const int warp_lo = p.window > 0 ? max(0, warp_min_pos - p.window + 1) : 0;
  const bool warp_full = warp_first + 15 < num_rows;
  const int krow = (lane & 7) + ((lane >> 4) << 3), kchunk = (lane >> 3) & 1;
  const int qrow = warp * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), qchunk = lane >> 4;
  const float scale2 = p.scale * 1.4426950408889634f;  // scores in log2 units

  int item = 0, kt0 = 0, tile = 0;
  bool live = false;
  for (int n = 0; n < total; ++n) {
    cp_async_wait<kPrefillStages - 2>();
    __syncthreads();
    load_next();
    if (item == 0) {
      kt0 = tiles.first_key(tile);
      live = kt0 <= warp_max_pos && (kt0 + kKeyTile > warp_lo || kt0 < p.keep);
#pragma unroll
      for (int j = 0; j < kKeyTile / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
    }
    if (live && item < p.KV) {
      const uint32_t k_tile = stage(n), q_part = kStreamQ ? k_tile + kTileBytes : q_all + (uint32_t)item * kQPart;
#pragma unroll
      for (int kc = 0; kc < HD / 16; ++kc) {
        uint32_t a[4];
        ldmatrix_x4(a, q_part + tile_offset<HD>(qrow, kc * 2 + qchunk));
#pragma unroll
        for (int g = 0; g < kKeyTile / 16; ++g) {
          uint32_t b[4];
          ldmatrix_x4(b, k_tile + tile_offset<HD>(g * 16 + krow, kc * 2 + kchunk));
          mma_bf16(s[g * 2], a, b[0], b[1]);
          mma_bf16(s[g * 2 + 1], a, b[2], b[3]);
        }
      }
    } else if (live) {
      const bool inside = warp_full && kt0 + kKeyTile <= warp_min_pos + 1 &&
                          (p.window <= 0 || kt0 > warp_max_pos - p.window || kt0 + kKeyTile <= p.keep);
      float rmax[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int j = 0; j < kKeyTile / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[j][e] *= scale2;
          if (!inside) {
            const int key = kt0 + j * 8 + (lane & 3) * 2 + (e & 1), qp = qpos[e >> 1];
            if (!(key <= qp && (p.window <= 0 || key > qp - p.window || key < p.keep))) s[j][e] = -INFINITY;
          }
          rmax[e >> 1] = fmaxf(rmax[e >> 1], s[j][e]);
        }
      float corr[2], rsum[2] = {0.f, 0.f}, m_use[2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        rmax[h] = fmaxf(rmax[h], __shfl_xor_sync(0xffffffffu, rmax[h], 1));
        rmax[h] = fmaxf(rmax[h], __shfl_xor_sync(0xffffffffu, rmax[h], 2));
        const float m_new = fmaxf(m[h], rmax[h]);
        m_use[h] = m_new == -INFINITY ? 0.f : m_new;  // a row that has seen nothing yet
        corr[h] = fast_exp2(m[h] - m_use[h]);
        m[h] = m_new;
      }
#pragma unroll
      for (int j = 0; j < kKeyTile / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[j][e] = fast_exp2(s[j][e] - m_use[e >> 1]);
          rsum[e >> 1] += s[j][e];
        }
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        rsum[h] += __shfl_xor_sync(0xffffffffu, rsum[h], 1);
        rsum[h] += __shfl_xor_sync(0xffffffffu, rsum[h], 2);
        l[h] = l[h] * corr[h] + rsum[h];
      }
#pragma unroll
      for (int i = 0; i < HD / 8; ++i) {
        acc[i][0] *= corr[0]; acc[i][1] *= corr[0];
        acc[i][2] *= corr[1]; acc[i][3] *= corr[1];
      }
#pragma unroll
      for (int g = 0; g < kKeyTile / 16; ++g) {
        const uint32_t pf[4] = {pack_bf16(s[g * 2][0], s[g * 2][1]), pack_bf16(s[g * 2][2], s[g * 2][3]),
                                pack_bf16(s[g * 2 + 1][0], s[g * 2 + 1][1]), pack_bf16(s[g * 2 + 1][2], s[g * 2 + 1][3])};
        pv_16keys<HD>(acc, pf, stage(n), g * 16, lane);
      }
    }
    if (++item == items) { item = 0; ++tile; }
  }
  cp_async_wait<0>();

#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int rr = warp * 16 + (lane >> 2) + h * 8;
    if (rr >= num_rows) continue;
    const int qi = rr / gc, g = rr - qi * gc;
    __nv_bfloat16* o = p.out + ((size_t)(row0 + qi) * p.H + head0 + g) * HD;
    const float inv = 1.f / l[h];
#pragma unroll
    for (int i = 0; i < HD / 8; ++i)
      *reinterpret_cast<__nv_bfloat162*>(o + i * 8 + (lane & 3) * 2) = __floats2bfloat162_rn(acc[i][h * 2] * inv, acc[i][h * 2 + 1] * inv);
  }
}

constexpr size_t kMaxSmem = 227 * 1024;

int decode_groups(int H) { return H > 16 ? 2 : 1; }
size_t decode_smem(int hd, int H, int KV, int stages) {
  return (size_t)stages * kKeyTile * hd * 2 + (size_t)KV * decode_groups(H) * 16 * hd * 2;
}
// four stages where two blocks then share an SM, else eight where they fit (one block keeps the copies going)
int decode_stages(int hd, int H, int KV) {
  return decode_smem(hd, H, KV, 4) > 113 * 1024 && decode_smem(hd, H, KV, 8) <= kMaxSmem ? 8 : 4;
}
// heads per block: whole groups where they fit its rows, so that no value head is read twice
int decode_heads(int H, int KV) {
  const int G = H / KV, most = 16 * decode_groups(H);
  return H <= most ? H : (G <= most ? most / G * G : most);
}
size_t prefill_smem(int hd, int KV, bool stream) {
  const size_t tile = (size_t)kKeyTile * hd * 2, q = (size_t)kPrefillRows * hd * 2;
  return stream ? kPrefillStages * (tile + q) : kPrefillStages * tile + KV * q;
}

template <typename Kernel>
int start(Kernel kern, dim3 grid, int threads, size_t smem, cudaStream_t stream, const PartsParams& p, const char* what) {
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return asb::fail("%s: shared memory %zu: %s", what, smem, cudaGetErrorString(e));
  asb::launch(kern, grid, threads, smem, stream, p);
  return asb::check_launch(what);
}

template <typename F>
auto with_decode_kernel(int hd, int H, int KV, F&& use) {
  const bool two = decode_groups(H) == 2, eight = decode_stages(hd, H, KV) == 8;
#define ASB_PICK(HD) \
  (two ? (eight ? use(parts_decode_kernel<HD, 2, 8>) : use(parts_decode_kernel<HD, 2, 4>)) \
       : (eight ? use(parts_decode_kernel<HD, 1, 8>) : use(parts_decode_kernel<HD, 1, 4>)))
  return hd == 64 ? ASB_PICK(64) : ASB_PICK(128);
#undef ASB_PICK
}

template <int HD>
int launch_parts(PartsParams p, int run_decode, int run_prefill, cudaStream_t stream) {
  if (run_decode) {
    p.GC = decode_heads(p.H, p.KV);
    p.HC = (p.H + p.GC - 1) / p.GC;
    if (p.HC > 65535) return asb::fail("attention_parts: too many heads");
    dim3 grid(p.short_rows > 0 ? p.short_rows : p.T, p.HC, p.NP);
    const size_t smem = decode_smem(HD, p.H, p.KV, decode_stages(HD, p.H, p.KV));
    if (int rc = with_decode_kernel(HD, p.H, p.KV, [&](auto kern) { return start(kern, grid, 128 * decode_groups(p.H), smem, stream, p, "parts_decode"); })) return rc;
  }
  if (run_prefill) {
    p.GC = p.G < 16 ? p.G : 16;
    p.HC = (p.G + p.GC - 1) / p.GC;
    p.QT = kPrefillRows / p.GC;
    const bool stream_q = prefill_smem(HD, p.KV, false) > kMaxSmem;
    const size_t smem = prefill_smem(HD, p.KV, stream_q);
    const long long blocks = (long long)((p.T + p.QT - 1) / p.QT + p.R) * p.KV * p.HC;
    if (blocks > 0x7fffffffLL) return asb::fail("attention_parts: %lld blocks exceed the grid", blocks);
    const dim3 grid((unsigned)blocks);
    if (stream_q) return start(parts_prefill_kernel<HD, true>, grid, kPrefillThreads, smem, stream, p, "parts_prefill");
    return start(parts_prefill_kernel<HD, false>, grid, kPrefillThreads, smem, stream, p, "parts_prefill");
  }
  return 0;
}

}  // namespace

// 1 if these kernels serve the shape: the decode kernel keeps a token's queries of all parts in shared memory.
extern "C" int asb_attention_parts_supported(int hd, int H, int KV) {
  return (hd == 64 || hd == 128) && KV >= 1 && decode_smem(hd, H, KV, 4) <= kMaxSmem ? 1 : 0;
}

// Query heads that share a block of the decode kernel, and blocks the device holds at once: for the
// caller's choice of partitions.
extern "C" int asb_attention_parts_heads(int H, int KV) { return decode_heads(H, KV); }
extern "C" int asb_attention_parts_resident(int hd, int H, int KV) {
  if (!asb_attention_parts_supported(hd, H, KV)) return 0;
  int device = 0, sms = 0, per_sm = 0;
  if (cudaGetDevice(&device) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device) != cudaSuccess) return 0;
  const size_t smem = decode_smem(hd, H, KV, decode_stages(hd, H, KV));
  const cudaError_t e = with_decode_kernel(hd, H, KV, [&](auto kern) {
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, kern, 128 * decode_groups(H), smem);
  });
  return e == cudaSuccess ? per_sm * sms : 0;
}

// q [T, H, KV, hd], out [T, H, hd]. Requests of at most 8 tokens go through the decode kernel
// (`run_decode`), longer ones through the prefill kernel. Partitions are PT key tiles of 64 each and
// apply to the decode kernel; with NP > 1 the caller merges the scratch with asb_attention_reduce
// (asb_attention_reduce_short where short_rows > 0: see attention_mma.cu).
extern "C" int asb_attention_parts(void* out, const void* q, const void* k_cache, const void* v_cache,
                                   const int* block_tables, const int* req_q_start, const int* req_pos_start,
                                   float* part_m, float* part_l, float* part_acc, int num_tokens, int R, int H, int KV,
                                   int hd, int bs, int table_width, int window, int keep, int PT, int NP, float scale,
                                   int run_decode, int run_prefill, int all_single, int short_rows, cudaStream_t stream) {
  if (num_tokens == 0 || R == 0) return 0;
  if (KV < 1 || H % KV) return asb::fail("attention_parts: %d heads over %d kv heads", H, KV);
  if (!asb_attention_parts_supported(hd, H, KV)) return asb::fail("attention_parts: head_dim %d with %d key heads is not served", hd, KV);
  if (window < 0 || keep < 0 || bs < 1) return asb::fail("attention_parts: window %d, keep %d, page %d", window, keep, bs);
  if (NP < 1 || NP > 65535 || PT < 1) return asb::fail("attention_parts: %d partitions of %d tiles", NP, PT);
  if (NP > 1 && (!part_m || !part_l || !part_acc)) return asb::fail("attention_parts: %d partitions need scratch", NP);
  if (short_rows < 0 || short_rows > num_tokens || (short_rows > 0 && all_single)) return asb::fail("attention_parts: %d short rows of %d tokens", short_rows, num_tokens);
  PartsParams p = {};
  p.q = (const __nv_bfloat16*)q; p.out = (__nv_bfloat16*)out;
  p.k_cache = (const __nv_bfloat16*)k_cache; p.v_cache = (const __nv_bfloat16*)v_cache;
  p.block_tables = block_tables; p.req_q_start = req_q_start; p.req_pos_start = req_pos_start;
  p.part_m = part_m; p.part_l = part_l; p.part_acc = part_acc;
  p.T = num_tokens; p.R = R; p.H = H; p.KV = KV; p.bs = bs; p.table_width = table_width; p.G = H / KV;
  p.window = window; p.keep = window > 0 ? keep : 0; p.PT = PT; p.NP = NP;
  p.all_single = all_single; p.short_rows = short_rows; p.scale = scale;
  if (hd == 64) return launch_parts<64>(p, run_decode, run_prefill, stream);
  return launch_parts<128>(p, run_decode, run_prefill, stream);
}
