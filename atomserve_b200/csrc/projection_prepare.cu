// What happens between an attention layer's stacked projection and its attention kernel where queries
// and keys are RMS-normed over their whole projection, all heads at once, before positions enter:
//
//   asb_projection_norm_rope_store   from one row [H * dim] q, [KV * dim] k, [KV * vdim] v of the
//       projection: q and k divided by their root mean squares over all their heads, times a gain per
//       column; the first `rotary_dim` entries of every head turned by position * inv_freq[i], entries i
//       and i + rotary_dim / 2 (or 2i and 2i + 1) being a pair; queries [T, H, hd], keys and values to
//       their pages as [KV, hd], zeros behind what a head holds (hd is the larger of dim and vdim).
//
// Sums, norms, angles and the rotation are float32; each stored value is rounded once.
#include "common.cuh"

namespace {

struct ProjectionParams {
  const void* proj;      // [T, stride], q from column q_off on, k and v behind it
  void* q_out;           // [T, H, hd]
  void* k_cache;         // [num_blocks, KV, bs, hd] or null: queries only
  void* v_cache;
  const float* q_gain;   // [H * dim]
  const float* k_gain;   // [KV * dim]
  const int* positions;  // [T]
  const int* slots;      // [T] page * bs + offset, -1: store nothing
  const float* inv_freq; // [rotary_dim / 2]
  int stride, q_off, H, KV, dim, vdim, hd, rotary_dim, interleaved, bs;
  float eps;
};

template <typename T, int VEC>
__device__ __forceinline__ void load_row(const T* at, float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    const uint4 raw = *reinterpret_cast<const uint4*>(at);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(h[i]);
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  } else if constexpr (VEC == 4) {
    const float4 f = *reinterpret_cast<const float4*>(at);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    v[0] = asb::to_float(at[0]);
  }
}

template <typename T, int VEC>
__device__ __forceinline__ void store_row(T* at, const float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(at) = raw;
  } else if constexpr (VEC == 4) {
    *reinterpret_cast<float4*>(at) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    at[0] = asb::from_float<T>(v[0]);
  }
}

// One block per token; VEC neighbouring entries a thread at a time (they share a head, and lie on one side
// of a rotation's halves). q and k wait in shared memory for their norms.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
projection_norm_rope_store_kernel(const ProjectionParams p) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float scratch[2][8];
  const int qw = p.H * p.dim, kw = p.KV * p.dim, half = p.rotary_dim >> 1, per = p.hd / VEC;
  float* row = smem;               // [qw + kw]
  float* cs = smem + qw + kw;      // [rotary_dim]: cosines, then sines
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const int t = blockIdx.x;
  const T* src = (const T*)p.proj + (size_t)t * p.stride + p.q_off;
  const float position = (float)p.positions[t];
  const int slot = p.slots ? p.slots[t] : -1;
  const bool store = p.k_cache && slot >= 0;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x * VEC; i < qw + (store ? kw : 0); i += 256 * VEC) {
    float v[VEC], ss = 0.f;
    load_row<T, VEC>(src + i, v);
#pragma unroll
    for (int u = 0; u < VEC; ++u) {
      row[i + u] = v[u];
      ss = fmaf(v[u], v[u], ss);
    }
    if (i < qw) sq += ss;
    else sk += ss;
  }
  for (int i = threadIdx.x; i < half; i += 256) sincosf(position * p.inv_freq[i], &cs[half + i], &cs[i]);
  sq = asb::warp_sum(sq);
  sk = asb::warp_sum(sk);
  if ((threadIdx.x & 31) == 0) {
    scratch[0][threadIdx.x >> 5] = sq;
    scratch[1][threadIdx.x >> 5] = sk;
  }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) {
    sq += scratch[0][w];
    sk += scratch[1][w];
  }
  const float inv_q = 1.f / sqrtf(sq / (float)qw + p.eps), inv_k = 1.f / sqrtf(sk / (float)kw + p.eps);
  const size_t page = store ? slot / p.bs : 0, off = store ? slot % p.bs : 0;
  T* q_out = (T*)p.q_out + (size_t)t * p.H * p.hd;
  const int heads = p.H + (store ? p.KV : 0);
  for (int i = threadIdx.x; i < heads * per; i += 256) {
    const int head = i / per, e = (i - head * per) * VEC;
    const bool query = head < p.H;
    const float* x = row + head * p.dim;  // (keys lie behind the queries)
    const float* gain = query ? p.q_gain + head * p.dim : p.k_gain + (head - p.H) * p.dim;
    const float inv = query ? inv_q : inv_k;
    float v[VEC];
#pragma unroll
    for (int u = 0; u < VEC; ++u) {
      const int at = e + u;
      float w = 0.f;
      if (at < p.dim) {
        w = x[at] * inv * gain[at];
        if (at < p.rotary_dim) {
          const int pair = p.interleaved ? at >> 1 : (at < half ? at : at - half);
          const int mate = p.interleaved ? at ^ 1 : (at < half ? at + half : at - half);
          const bool first = p.interleaved ? !(at & 1) : at < half;
          const float other = x[mate] * inv * gain[mate], c = cs[pair], s = cs[half + pair];
          w = first ? w * c - other * s : w * c + other * s;
        }
      }
      v[u] = w;
    }
    T* dst = query ? q_out + head * p.hd + e
                   : (T*)p.k_cache + ((page * p.KV + head - p.H) * p.bs + off) * p.hd + e;
    store_row<T, VEC>(dst, v);
  }
  if (!store) return;
  for (int i = threadIdx.x; i < p.KV * per; i += 256) {
    const int head = i / per, e = (i - head * per) * VEC;
    float v[VEC];
#pragma unroll
    for (int u = 0; u < VEC; ++u) v[u] = 0.f;
    if (e < p.vdim) load_row<T, VEC>(src + qw + kw + head * p.vdim + e, v);
    store_row<T, VEC>((T*)p.v_cache + ((page * p.KV + head) * p.bs + off) * p.hd + e, v);
  }
}

// The usual form (bfloat16, pairs of halves): a thread keeps units of two vectors of eight entries in
// registers from the projection to where they belong: the entries of a unit's first vector and those of its
// second are pairs, or, past the rotated entries, neighbours that only take their norm. kPer: units a thread.
template <int kPer>
__global__ void __launch_bounds__(256)
projection_norm_rope_store_units_kernel(const ProjectionParams p) {
  using T = __nv_bfloat16;
  extern __shared__ __align__(16) float cs[];  // [rotary_dim]: cosines, then sines
  __shared__ float scratch[2][8];
  const int qw = p.H * p.dim, kw = p.KV * p.dim, half = p.rotary_dim >> 1, turned = half >> 3, per = p.dim >> 4;
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const int t = blockIdx.x, nwarps = blockDim.x >> 5;
  const T* src = (const T*)p.proj + (size_t)t * p.stride + p.q_off;
  const float position = (float)p.positions[t];
  const int slot = p.slots ? p.slots[t] : -1;
  const bool store = p.k_cache && slot >= 0;
  const int units = (p.H + (store ? p.KV : 0)) * per;
  float a[kPer][8], b[kPer][8];
#pragma unroll
  for (int u = 0; u < kPer; ++u) {
    const int i = threadIdx.x + u * blockDim.x;
    if (i >= units) continue;
    const int head = i / per, w = i - head * per;
    const int e = w < turned ? w * 8 : p.rotary_dim + (w - turned) * 16;
    load_row<T, 8>(src + head * p.dim + e, a[u]);
    load_row<T, 8>(src + head * p.dim + e + (w < turned ? half : 8), b[u]);
  }
  for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(position * p.inv_freq[i], &cs[half + i], &cs[i]);
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int u = 0; u < kPer; ++u) {
    const int i = threadIdx.x + u * blockDim.x;
    if (i >= units) continue;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(a[u][j], a[u][j], fmaf(b[u][j], b[u][j], ss));
    if (i < p.H * per) sq += ss;
    else sk += ss;
  }
  sq = asb::warp_sum(sq);
  sk = asb::warp_sum(sk);
  if ((threadIdx.x & 31) == 0) {
    scratch[0][threadIdx.x >> 5] = sq;
    scratch[1][threadIdx.x >> 5] = sk;
  }
  __syncthreads();  // (the angles too)
  sq = sk = 0.f;
  for (int w = 0; w < nwarps; ++w) {
    sq += scratch[0][w];
    sk += scratch[1][w];
  }
  const float inv_q = 1.f / sqrtf(sq / (float)qw + p.eps), inv_k = 1.f / sqrtf(sk / (float)kw + p.eps);
  const size_t page = store ? slot / p.bs : 0, off = store ? slot % p.bs : 0;
#pragma unroll
  for (int u = 0; u < kPer; ++u) {
    const int i = threadIdx.x + u * blockDim.x;
    if (i >= units) continue;
    const int head = i / per, w = i - head * per;
    const bool query = head < p.H;
    const int e = w < turned ? w * 8 : p.rotary_dim + (w - turned) * 16, f = e + (w < turned ? half : 8);
    const float* gain = query ? p.q_gain + head * p.dim : p.k_gain + (head - p.H) * p.dim;
    const float inv = query ? inv_q : inv_k;
    float ga[8], gb[8];
#pragma unroll
    for (int j = 0; j < 8; j += 4) {
      *reinterpret_cast<float4*>(ga + j) = *reinterpret_cast<const float4*>(gain + e + j);
      *reinterpret_cast<float4*>(gb + j) = *reinterpret_cast<const float4*>(gain + f + j);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      a[u][j] *= inv * ga[j];
      b[u][j] *= inv * gb[j];
    }
    if (w < turned) {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float c = cs[e + j], s = cs[half + e + j], x = a[u][j], y = b[u][j];
        a[u][j] = x * c - y * s;
        b[u][j] = y * c + x * s;
      }
    }
    T* dst = query ? (T*)p.q_out + ((size_t)t * p.H + head) * p.hd : (T*)p.k_cache + ((page * p.KV + head - p.H) * p.bs + off) * p.hd;
    store_row<T, 8>(dst + e, a[u]);
    store_row<T, 8>(dst + f, b[u]);
  }
  const uint4 zero = make_uint4(0, 0, 0, 0);
  const int kz = (p.hd - p.dim) >> 3, per_v = p.hd >> 3;
  for (int i = threadIdx.x; i < (p.H + (store ? p.KV : 0)) * kz; i += blockDim.x) {  // zeros behind queries and keys
    const int head = i / kz, e = p.dim + i % kz * 8;
    T* dst = head < p.H ? (T*)p.q_out + ((size_t)t * p.H + head) * p.hd : (T*)p.k_cache + ((page * p.KV + head - p.H) * p.bs + off) * p.hd;
    *reinterpret_cast<uint4*>(dst + e) = zero;
  }
  if (!store) return;
  for (int i = threadIdx.x; i < p.KV * per_v; i += blockDim.x) {
    const int head = i / per_v, e = (i - head * per_v) * 8;
    *reinterpret_cast<uint4*>((T*)p.v_cache + ((page * p.KV + head) * p.bs + off) * p.hd + e) =
        e < p.vdim ? *reinterpret_cast<const uint4*>(src + qw + kw + head * p.vdim + e) : zero;
  }
}

template <typename T, int VEC>
int launch(const ProjectionParams& p, int T_, cudaStream_t stream) {
  const size_t smem = sizeof(float) * ((size_t)(p.H + p.KV) * p.dim + p.rotary_dim);
  auto kern = projection_norm_rope_store_kernel<T, VEC>;
  if (smem > 48 * 1024) {
    if (smem > 200 * 1024) return asb::fail("projection_norm_rope_store: %d + %d heads of %d do not fit shared memory", p.H, p.KV, p.dim);
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return asb::fail("projection_norm_rope_store: shared memory %zu: %s", smem, cudaGetErrorString(e));
  }
  asb::launch(kern, T_, 256, smem, stream, p);
  return asb::check_launch("projection_norm_rope_store");
}

}  // namespace

extern "C" int asb_projection_norm_rope_store(const void* proj, int stride, int q_off, void* q_out, void* k_cache, void* v_cache,
                                              const float* q_gain, const float* k_gain, const int* positions, const int* slots,
                                              const float* inv_freq, int T_, int H, int KV, int dim, int vdim, int hd, int rotary_dim,
                                              int interleaved, int bs, float eps, int dtype, cudaStream_t stream) {
  if (T_ == 0) return 0;
  if (H < 1 || KV < 1 || dim < 1 || vdim < 1 || dim > hd || vdim > hd) return asb::fail("projection_norm_rope_store: keys of %d and values of %d in heads of %d", dim, vdim, hd);
  if (rotary_dim % 2 || rotary_dim < 0 || rotary_dim > dim || (rotary_dim && !inv_freq)) return asb::fail("projection_norm_rope_store: rotary_dim %d against dim %d", rotary_dim, dim);
  if (q_off < 0 || stride < q_off + H * dim + (k_cache ? KV * (dim + vdim) : 0)) return asb::fail("projection_norm_rope_store: rows of %d hold no such projection", stride);
  if (k_cache && (!v_cache || !slots || bs < 1)) return asb::fail("projection_norm_rope_store: pages need values, slots and a page size");
  ProjectionParams p;
  p.proj = proj; p.q_out = q_out; p.k_cache = k_cache; p.v_cache = v_cache; p.q_gain = q_gain; p.k_gain = k_gain;
  p.positions = positions; p.slots = slots; p.inv_freq = inv_freq; p.stride = stride; p.q_off = q_off; p.H = H; p.KV = KV;
  p.dim = dim; p.vdim = vdim; p.hd = hd; p.rotary_dim = rotary_dim; p.interleaved = interleaved; p.bs = bs; p.eps = eps;
  const bool aligned = (((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) == 0;
  const int vec = dtype == asb::kBFloat16 ? 8 : 4;
  if (aligned && dim % vec == 0 && vdim % vec == 0 && stride % vec == 0 && q_off % vec == 0) {
    const int units = (H + KV) * (dim / 16);
    if (dtype == asb::kBFloat16 && !interleaved && dim % 16 == 0 && rotary_dim % 16 == 0 && units <= 1024 &&
        (((uintptr_t)q_gain | (uintptr_t)k_gain) & 15) == 0) {
      const int threads = units >= 256 ? 256 : (units + 31) / 32 * 32;
      const size_t smem = sizeof(float) * (rotary_dim > 0 ? rotary_dim : 1);
      if (units <= 256) asb::launch(projection_norm_rope_store_units_kernel<1>, T_, threads, smem, stream, p);
      else if (units <= 512) asb::launch(projection_norm_rope_store_units_kernel<2>, T_, threads, smem, stream, p);
      else asb::launch(projection_norm_rope_store_units_kernel<4>, T_, threads, smem, stream, p);
      return asb::check_launch("projection_norm_rope_store");
    }
    if (dtype == asb::kBFloat16) return launch<__nv_bfloat16, 8>(p, T_, stream);
    if (dtype == asb::kFloat32) return launch<float, 4>(p, T_, stream);
  }
  ASB_DISPATCH_DTYPE(dtype, T, { return launch<T, 1>(p, T_, stream); });
  return 0;
}
