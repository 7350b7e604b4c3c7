// What happens between an attention layer's stacked projection and its attention kernel where every
// head's score is a mix of all heads' scores before the softmax ("talking heads"),
//
//   score_h(i, j) = sum_g talk[h, g] q_g(i) . k_c(g)(j),   c(g) the kv head that head g reads.
//
// The mix is linear in the queries, so it moves into them: with q'[h, c] = sum over the heads g of kv
// head c of talk[h, g] q_g, a head's score is sum_c q'[h, c] . k_c, and the paged attention kernels
// serve heads of KV key parts (attention_simt.cu, attention_parts.cu, attention_parts_tcgen05.cu). No
// score is ever rounded between the product and the mix.
//
//   asb_mixed_heads_prepare   from one row [H * dim] q, [KV * dim] k, [KV * vdim] v of the projection:
//       add the biases; RMS-norm q over all its heads at once, and k (gains per entry); turn the
//       first `rotary_dim` entries of every head by position * inv_freq[i], entries 2i and 2i + 1
//       (or i and i + rotary_dim / 2) being a pair; write
//         q' [T, H, KV, hd]: each part's `dim` entries, then zeros,
//         keys to their page as [KV, hd], then zeros,
//         values to their page as [KV, hd]: v, or (1 - lambda) v + lambda v_first of the same token
//         where the layer mixes its values with an earlier layer's, then zeros,
//         and v itself as a tensor [T, KV * vdim] where later layers will want it as their v_first.
//       Without pages only the queries are made. The projection may come as the partial sums that
//       the tensor-core GEMM left in its workspace (few tokens).
//
// Sums, norms, angles, sines, the rotation, the mix of the queries and of the values are float32;
// each stored value is rounded once.
#include "common.cuh"
#include "gemm_partials.cuh"

namespace {

struct MixedParams {
  const void* proj;   // [T, row], or null: partial sums
  asb::PartialSums ps;
  const float* bias;  // [H * dim + KV * dim + KV * vdim] or null
  const float* q_gain;  // [H * dim] or null: no norms
  const float* k_gain;  // [KV * dim]
  const float* talk;  // [H, H]
  const void* v_first;  // [T, KV * vdim] or null
  void* v_out;        // [T, KV * vdim] or null
  void* q_out;        // [T, H, KV, hd]
  void* k_cache;      // [num_blocks, KV, bs, hd] or null
  void* v_cache;
  const int* positions;  // [T]
  const int* slots;      // [T] page * bs + offset, -1: store nothing
  const float* inv_freq; // [rotary_dim / 2]
  int H, KV, dim, vdim, hd, rotary_dim, bs, row, interleaved;
  float eps, lambda;
};

template <typename T>
__device__ __forceinline__ void store4(T* at, const float (&v)[4]) {
  if constexpr (sizeof(T) == 2) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(at) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
  } else {
    *reinterpret_cast<float4*>(at) = make_float4(v[0], v[1], v[2], v[3]);
  }
}
template <typename T>
__device__ __forceinline__ void load4(const T* at, float (&v)[4]) {
  if constexpr (sizeof(T) == 2) {
    const uint2 raw = *reinterpret_cast<const uint2*>(at);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  } else {
    const float4 f = *reinterpret_cast<const float4*>(at);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  }
}

// V neighbouring columns of a token's projection, bias added
template <typename T, int V>
__device__ __forceinline__ void column(const MixedParams& p, int t, int col, float (&v)[V], bool biased = true) {
  if (p.proj) {
    const T* at = (const T*)p.proj + (size_t)t * p.row + col;
    if constexpr (V == 4) {
      load4<T>(at, v);
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) v[k] = asb::to_float(at[k]);
    }
  } else {
    asb::partial_sum<V>(p.ps, t, col, asb::partial_slots(p.ps, col / asb::kPartialRows), v);
  }
  if (biased && p.bias) {
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] += p.bias[col + k];
  }
}

template <typename T>
__device__ __forceinline__ void store8(T* at, const float (&v)[8]) {
  if constexpr (sizeof(T) == 2) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(at) = raw;
  } else {
    *reinterpret_cast<float4*>(at) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>((float*)at + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
}

// `heads` heads of `dim` columns from `col` on into dst [heads][hd]; returns the thread's sum of squares
template <typename T, int V>
__device__ __forceinline__ float gather_heads(const MixedParams& p, int t, int col, int heads, int dim, float* dst) {
  float ss = 0.f;
  const int per = dim / V;  // (V divides dim)
  for (int i = threadIdx.x; i < heads * per; i += blockDim.x) {
    const int h = i / per, e = (i - h * per) * V;
    float v[V];
    column<T, V>(p, t, col + h * dim + e, v);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      dst[h * p.hd + e + k] = v[k];
      ss = fmaf(v[k], v[k], ss);
    }
  }
  return ss;
}

// norm (inv = 1 / rms, gains per entry) and rotation of heads in place; a thread owns both entries of a pair
__device__ __forceinline__ void norm_and_turn(const MixedParams& p, float* x, int heads, const float* gain, float inv, const float* cs) {
  const int half = p.rotary_dim >> 1, units = half + (p.dim - p.rotary_dim);
  for (int i = threadIdx.x; i < heads * units; i += blockDim.x) {
    const int h = i / units, u = i - h * units;
    float* head = x + h * p.hd;
    const float* g = gain ? gain + h * p.dim : nullptr;
    if (u < half) {
      const int a = p.interleaved ? 2 * u : u, b = p.interleaved ? 2 * u + 1 : u + half;
      float va = head[a], vb = head[b];
      if (g) { va = va * inv * g[a]; vb = vb * inv * g[b]; }
      const float c = cs[u], s = cs[half + u];
      head[a] = va * c - vb * s;
      head[b] = vb * c + va * s;
    } else if (g) {
      const int e = p.rotary_dim + (u - half);
      head[e] = head[e] * inv * g[e];
    }
  }
}

// The general form: any sizes, both pairings. One block per token; V: columns read at a time.
template <typename T, int V>
__global__ void __launch_bounds__(256)
mixed_heads_prepare_kernel(const MixedParams p) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float scratch[32];
  const int H = p.H, KV = p.KV, hd = p.hd, dim = p.dim, G = H / KV;
  float* q_s = smem;                // [H][hd], zeros behind dim
  float* k_s = q_s + H * hd;        // [KV][hd]
  float* talk_s = k_s + KV * hd;    // [H][H]
  float* cs = talk_s + H * H;       // [rotary_dim] cosines, then sines
  // what no kernel writes is read before the wait
  for (int i = threadIdx.x; i < H * H; i += blockDim.x) talk_s[i] = p.talk[i];
  if (dim < hd) {
    for (int i = threadIdx.x; i < (H + KV) * (hd - dim); i += blockDim.x) {
      const int h = i / (hd - dim);
      smem[h * hd + dim + (i - h * (hd - dim))] = 0.f;
    }
  }
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const int t = blockIdx.x;
  const int half = p.rotary_dim >> 1;
  const float position = (float)__ldcg(p.positions + t);
  for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(position * p.inv_freq[i], &cs[half + i], &cs[i]);
  const int k_col = H * dim, v_col = k_col + KV * dim;
  const int slot = p.slots ? __ldcg(p.slots + t) : -1;
  const bool store = p.k_cache && slot >= 0;
  const float sq = gather_heads<T, V>(p, t, 0, H, dim, q_s);
  const float sk = store ? gather_heads<T, V>(p, t, k_col, KV, dim, k_s) : 0.f;
  float inv_q = 1.f, inv_k = 1.f;
  if (p.q_gain) {
    inv_q = 1.f / sqrtf(asb::block_sum(sq, scratch) / (float)(H * dim) + p.eps);
    inv_k = 1.f / sqrtf(asb::block_sum(sk, scratch) / (float)(KV * dim) + p.eps);
  }
  __syncthreads();
  norm_and_turn(p, q_s, H, p.q_gain, inv_q, cs);
  if (store) norm_and_turn(p, k_s, KV, p.k_gain, inv_k, cs);

  // values: biased, mixed, to their page
  const size_t page = store ? slot / p.bs : 0, off = store ? slot % p.bs : 0;
  if (p.k_cache) {
    const int per = p.vdim / V;
    for (int i = threadIdx.x; i < KV * per; i += blockDim.x) {
      const int c = i / per, e = (i - c * per) * V;
      float v[V];
      column<T, V>(p, t, v_col + c * p.vdim + e, v);
      const size_t at = (size_t)t * KV * p.vdim + c * p.vdim + e;
#pragma unroll
      for (int k = 0; k < V; ++k) {
        const T own = asb::from_float<T>(v[k]);
        if (p.v_out) ((T*)p.v_out)[at + k] = own;
        T kept = own;
        if (p.v_first) kept = asb::from_float<T>((1.f - p.lambda) * v[k] + p.lambda * asb::to_float(((const T*)p.v_first)[at + k]));
        if (store) ((T*)p.v_cache)[((page * KV + c) * p.bs + off) * hd + e + k] = kept;
      }
    }
    if (store)
      for (int i = threadIdx.x; i < KV * (hd - p.vdim); i += blockDim.x) {
        const int c = i / (hd - p.vdim), e = p.vdim + (i - c * (hd - p.vdim));
        ((T*)p.v_cache)[((page * KV + c) * p.bs + off) * hd + e] = asb::from_float<T>(0.f);
      }
  }
  __syncthreads();
  T* q_out = (T*)p.q_out + (size_t)t * H * KV * hd;
  if (store)
    for (int i = threadIdx.x; i < KV * hd; i += blockDim.x) {
      const int c = i / hd, e = i - c * hd;
      ((T*)p.k_cache)[((page * KV + c) * p.bs + off) * hd + e] = asb::from_float<T>(k_s[i]);
    }
  for (int i = threadIdx.x; i < H * KV * hd; i += blockDim.x) {
    const int e = i % hd, hc = i / hd, c = hc % KV, h = hc / KV;
    float v = 0.f;
    for (int g = c * G; g < (c + 1) * G; ++g) v = fmaf(talk_s[h * H + g], q_s[g * hd + e], v);
    q_out[i] = asb::from_float<T>(v);
  }
}

// The usual form: neighbouring pairs (or no rotation), head sizes that are multiples of 8. A thread keeps
// its vectors of four columns in registers from the projection to where they belong: both entries of a
// pair lie in one vector, so norm and rotation touch no shared memory; keys and values go to their
// pages and queries to shared memory for the mix. kPer: vectors a thread. R and E: the group's heads
// whose E entries a thread holds while it walks the output heads.
template <typename T, int R, int E, int kPer>
__global__ void __launch_bounds__(256, kPer <= 6 ? 3 : 2)
mixed_heads_prepare_vec_kernel(const MixedParams p) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float scratch[2][8];
  const int H = p.H, KV = p.KV, hd = p.hd, dim = p.dim;
  float* q_s = smem;              // [H][hd], zeros behind dim
  float* talk_s = q_s + H * hd;   // [H][H]
  float* cs = talk_s + H * H;     // [rotary_dim] cosines, then sines
  const int nq = H * dim >> 2, nk = KV * dim >> 2, nv = p.k_cache ? KV * p.vdim >> 2 : 0, total = nq + (p.k_cache ? nk + nv : 0);
  // what no kernel writes is read before the wait
  for (int i = threadIdx.x; i < H * H; i += 256) talk_s[i] = p.talk[i];
  for (int i = threadIdx.x; i < H * (hd - dim); i += 256) q_s[i / (hd - dim) * hd + dim + i % (hd - dim)] = 0.f;
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const int half = p.rotary_dim >> 1;
  const int t = blockIdx.x;
  float v[kPer][4];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int u = 0; u < kPer; ++u) {
    const int i = threadIdx.x + u * 256;
    if (i < total) column<T, 4>(p, t, 4 * i, v[u], false);
  }
  const float position = (float)__ldcg(p.positions + t);
  for (int i = threadIdx.x; i < half; i += 256) sincosf(position * p.inv_freq[i], &cs[half + i], &cs[i]);
  const int slot = p.slots ? __ldcg(p.slots + t) : -1;
  const bool store = p.k_cache && slot >= 0;
#pragma unroll
  for (int u = 0; u < kPer; ++u) {
    const int i = threadIdx.x + u * 256;
    if (i >= total) continue;
    if (p.bias) {
      const float4 b = *reinterpret_cast<const float4*>(p.bias + 4 * i);
      v[u][0] += b.x; v[u][1] += b.y; v[u][2] += b.z; v[u][3] += b.w;
    }
    const float ss = v[u][0] * v[u][0] + v[u][1] * v[u][1] + v[u][2] * v[u][2] + v[u][3] * v[u][3];
    if (i < nq) sq += ss;
    else if (i < nq + nk) sk += ss;
  }
  sq = asb::warp_sum(sq);
  sk = asb::warp_sum(sk);
  if ((threadIdx.x & 31) == 0) {
    scratch[0][threadIdx.x >> 5] = sq;
    scratch[1][threadIdx.x >> 5] = sk;
  }
  __syncthreads();  // (the angles too)
  float inv_q = 1.f, inv_k = 1.f;
  if (p.q_gain) {
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      sq += scratch[0][w];
      sk += scratch[1][w];
    }
    inv_q = 1.f / sqrtf(sq / (float)(H * dim) + p.eps);
    inv_k = 1.f / sqrtf(sk / (float)(KV * dim) + p.eps);
  }
  const size_t page = store ? slot / p.bs : 0, off = store ? slot % p.bs : 0;
#pragma unroll
  for (int u = 0; u < kPer; ++u) {
    const int i = threadIdx.x + u * 256;
    if (i >= total) continue;
    if (i < nq + nk) {
      const bool query = i < nq;
      const int col = 4 * (query ? i : i - nq), h = col / dim, e = col - h * dim;
      float w[4] = {v[u][0], v[u][1], v[u][2], v[u][3]};
      if (p.q_gain) {
        const float4 g = *reinterpret_cast<const float4*>((query ? p.q_gain : p.k_gain) + col);
        const float inv = query ? inv_q : inv_k;
        w[0] *= inv * g.x; w[1] *= inv * g.y; w[2] *= inv * g.z; w[3] *= inv * g.w;
      }
#pragma unroll
      for (int k = 0; k < 4; k += 2) {
        const int pair = (e + k) >> 1;
        if (pair < half) {
          const float c = cs[pair], s = cs[half + pair], a = w[k], b = w[k + 1];
          w[k] = a * c - b * s;
          w[k + 1] = b * c + a * s;
        }
      }
      if (query) *reinterpret_cast<float4*>(q_s + h * hd + e) = make_float4(w[0], w[1], w[2], w[3]);
      else if (store) store4<T>((T*)p.k_cache + ((page * KV + h) * p.bs + off) * hd + e, w);
    } else {
      const int col = 4 * (i - nq - nk), h = col / p.vdim, e = col - h * p.vdim;
      const size_t at = (size_t)t * KV * p.vdim + col;
      if (p.v_out) store4<T>((T*)p.v_out + at, v[u]);
      if (p.v_first) {
        float f[4];
        load4<T>((const T*)p.v_first + at, f);
#pragma unroll
        for (int k = 0; k < 4; ++k) v[u][k] = (1.f - p.lambda) * v[u][k] + p.lambda * f[k];
      }
      if (store) store4<T>((T*)p.v_cache + ((page * KV + h) * p.bs + off) * hd + e, v[u]);
    }
  }
  if (store) {  // zeros behind what a head holds
    const float zero[4] = {0.f, 0.f, 0.f, 0.f};
    const int kz = (hd - dim) >> 2, vz = (hd - p.vdim) >> 2;
    for (int i = threadIdx.x; i < KV * kz; i += 256) store4<T>((T*)p.k_cache + ((page * KV + i / kz) * p.bs + off) * hd + dim + i % kz * 4, zero);
    for (int i = threadIdx.x; i < KV * vz; i += 256) store4<T>((T*)p.v_cache + ((page * KV + i / vz) * p.bs + off) * hd + p.vdim + i % vz * 4, zero);
  }
  __syncthreads();
  T* q_out = (T*)p.q_out + (size_t)t * H * KV * hd;
  // (part, E entries) per thread; the threads that are left over share the output heads
  const int per = hd / E, items = KV * per, lanes = items < 256 ? 256 / items : 1;
  for (int item = (int)threadIdx.x < items * lanes ? threadIdx.x % items : items; item < items; item += 256) {
    const int c = item / per, e = (item - c * per) * E;
    float q[R][E];
#pragma unroll
    for (int g = 0; g < R; ++g)
#pragma unroll
      for (int k = 0; k < E; k += 4) {
        const float4 f = *reinterpret_cast<const float4*>(q_s + (c * R + g) * hd + e + k);
        q[g][k] = f.x; q[g][k + 1] = f.y; q[g][k + 2] = f.z; q[g][k + 3] = f.w;
      }
    for (int h = items < 256 ? threadIdx.x / items : 0; h < H; h += lanes) {
      float sum[E], w[R];
#pragma unroll
      for (int g = 0; g < R; g += R >= 4 ? 4 : 1) {
        const float* at = talk_s + h * H + c * R + g;
        if constexpr (R >= 4) {
          const float4 f = *reinterpret_cast<const float4*>(at);
          w[g] = f.x; w[g + 1] = f.y; w[g + 2] = f.z; w[g + 3] = f.w;
        } else {
          w[g] = *at;
        }
      }
#pragma unroll
      for (int k = 0; k < E; ++k) sum[k] = 0.f;
#pragma unroll
      for (int g = 0; g < R; ++g)
#pragma unroll
        for (int k = 0; k < E; ++k) sum[k] = fmaf(w[g], q[g][k], sum[k]);
      T* at = q_out + ((size_t)h * KV + c) * hd + e;
      if constexpr (E == 8) store8<T>(at, sum);
      else store4<T>(at, sum);
    }
  }
}

template <typename Kernel>
int start(Kernel kern, const MixedParams& p, int tokens, size_t smem, cudaStream_t stream) {
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return asb::fail("mixed_heads_prepare: shared memory %zu: %s", smem, cudaGetErrorString(e));
  asb::launch(kern, tokens, 256, smem, stream, p);
  return asb::check_launch("mixed_heads_prepare");
}

template <typename T, int R, int E>
int start_vec(const MixedParams& p, int tokens, int vectors, size_t smem, cudaStream_t stream) {
  if (vectors <= 3 * 256) return start(mixed_heads_prepare_vec_kernel<T, R, E, 3>, p, tokens, smem, stream);
  if (vectors <= 6 * 256) return start(mixed_heads_prepare_vec_kernel<T, R, E, 6>, p, tokens, smem, stream);
  return start(mixed_heads_prepare_vec_kernel<T, R, E, 8>, p, tokens, smem, stream);
}

template <typename T>
int dispatch(const MixedParams& p, int tokens, cudaStream_t stream) {
  const size_t smem = sizeof(float) * ((size_t)(p.H + p.KV) * p.hd + (size_t)p.H * p.H + p.rotary_dim + 4);
  if (smem > 220 * 1024) return asb::fail("mixed_heads_prepare: %d heads of %d need %zu bytes of shared memory", p.H, p.hd, smem);
  const int G = p.H / p.KV, vectors = (p.H * p.dim + p.KV * (p.dim + p.vdim)) / 4;
  const bool four = p.dim % 4 == 0 && p.vdim % 4 == 0 && p.row % 4 == 0 &&
                    (((uintptr_t)p.proj | (uintptr_t)p.ps.ws) & 15) == 0;
  const bool eight = four && p.hd % 8 == 0 && vectors <= 8 * 256 && (p.interleaved || p.rotary_dim == 0) &&
                     (((uintptr_t)p.q_out | (uintptr_t)p.k_cache | (uintptr_t)p.v_cache | (uintptr_t)p.v_first | (uintptr_t)p.v_out |
                       (uintptr_t)p.bias | (uintptr_t)p.q_gain | (uintptr_t)p.k_gain) & 15) == 0;
  if (eight && G == 1) return start_vec<T, 1, 8>(p, tokens, vectors, smem, stream);
  if (eight && G == 2) return start_vec<T, 2, 8>(p, tokens, vectors, smem, stream);
  if (eight && G == 4) return start_vec<T, 4, 8>(p, tokens, vectors, smem, stream);
  if (eight && G == 8) return start_vec<T, 8, 4>(p, tokens, vectors, smem, stream);
  if (four) return start(mixed_heads_prepare_kernel<T, 4>, p, tokens, smem, stream);
  return start(mixed_heads_prepare_kernel<T, 1>, p, tokens, smem, stream);
}

}  // namespace

// proj [T, row] in `dtype`, or null with the partial sums of asb_gemm_tcgen05 mode 3 (bfloat16 outputs).
extern "C" int asb_mixed_heads_prepare(const void* proj, const float* ws, int max_slots, int bn, int kb_per_tile,
                                       int num_tiles, int blocks, const float* bias, const float* q_gain,
                                       const float* k_gain, const float* talk, const void* v_first, void* v_out,
                                       void* q_out, void* k_cache, void* v_cache, const int* positions, const int* slots,
                                       const float* inv_freq, int T_, int row, int H, int KV, int dim, int vdim, int hd,
                                       int rotary_dim, int interleaved, int bs, float eps, float lambda, int dtype,
                                       cudaStream_t stream) {
  if (T_ == 0) return 0;
  if (KV < 1 || H < 1 || H % KV) return asb::fail("mixed_heads_prepare: %d heads over %d kv heads", H, KV);
  if (dim < 1 || vdim < 1 || dim > hd || vdim > hd) return asb::fail("mixed_heads_prepare: keys of %d and values of %d do not fit heads of %d", dim, vdim, hd);
  if (rotary_dim % 2 || rotary_dim < 0 || rotary_dim > dim || (rotary_dim && !inv_freq)) return asb::fail("mixed_heads_prepare: rotary_dim %d against dim %d", rotary_dim, dim);
  const int columns = H * dim + (k_cache ? KV * (dim + vdim) : 0);
  if (proj ? row < columns : (!ws || T_ > bn || num_tiles * asb::kPartialRows < columns || dtype != asb::kBFloat16))
    return asb::fail("mixed_heads_prepare: rows of %d hold no such projection", row);
  if (k_cache && (!v_cache || !slots || bs < 1)) return asb::fail("mixed_heads_prepare: pages need values, slots and a page size");
  if ((q_gain != nullptr) != (k_gain != nullptr)) return asb::fail("mixed_heads_prepare: queries and keys are normed together or not at all");
  MixedParams p;
  p.proj = proj; p.ps = asb::PartialSums{ws, max_slots, bn, kb_per_tile, num_tiles, blocks};
  p.bias = bias; p.q_gain = q_gain; p.k_gain = k_gain; p.talk = talk; p.v_first = v_first; p.v_out = v_out;
  p.q_out = q_out; p.k_cache = k_cache; p.v_cache = v_cache; p.positions = positions; p.slots = slots; p.inv_freq = inv_freq;
  p.H = H; p.KV = KV; p.dim = dim; p.vdim = vdim; p.hd = hd; p.rotary_dim = rotary_dim; p.bs = bs;
  p.row = proj ? row : 0; p.interleaved = interleaved; p.eps = eps; p.lambda = lambda;
  ASB_DISPATCH_DTYPE(dtype, T, return dispatch<T>(p, T_, stream));
  return 0;
}
