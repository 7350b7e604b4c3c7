// Kernels for models whose layers add two sublayers that read the same stream,
// x <- x + mult (mixer(N1 x) + ff(N2 x)), over a float32 residual stream, and for what such a
// model does around its layers:
//
//   asb_residual_terms_norm  s = x + sum_i f_i y_i + bias (up to four terms, x and bias optional),
//                            written as the float32 stream, and N(s) gain1, N(s) gain2 in the compute
//                            dtype, N(s) = s / sqrt(mean(s^2) + eps): the sum of a layer, whatever
//                            number of outputs it has, and both norms of the next one in one pass
//   asb_partial_residual_terms_norm  the same with one more term given as the partial sums that the
//                            tensor-core GEMM left in its workspace (few tokens): a thread adds up the
//                            slots of 8 columns itself, in the order of the GEMM's own reduction
//   asb_pair_embedding       x[t] = table[id[t]] + pairs[row(previous id, id[t])], float32: a
//                            hashed table of token pairs beside the token table. The id before a
//                            request's first token of the step is per-request state (0: none yet)
//   asb_concat_cast          [a ; b] per row in the compute dtype (the input of a product over
//                            two streams)
//
// Sums and norms are float32; each stored value is rounded once.
#include "common.cuh"
#include "gemm_partials.cuh"

namespace {

int threads_for(int width) {
  int threads = 64;
  while (threads < width && threads < 1024) threads <<= 1;
  return threads;
}

constexpr int kMaxTerms = 4;
struct Terms {
  const float* y[kMaxTerms];
  float f[kMaxTerms];
  int n;
};

// One block per row; the row's sum stays in shared memory between the two passes.
template <typename T>
__global__ void residual_terms_norm_kernel(float* __restrict__ out32, T* __restrict__ out1, T* __restrict__ out2,
                                           const float* __restrict__ x, const Terms terms, const float* __restrict__ bias,
                                           const float* __restrict__ gain1, const float* __restrict__ gain2, int width, float eps) {
  extern __shared__ float row[];
  __shared__ float scratch[32];
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const size_t at = (size_t)blockIdx.x * width;
  float ss = 0.f;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    float s = x ? x[at + i] : 0.f;
#pragma unroll
    for (int u = 0; u < kMaxTerms; ++u)
      if (u < terms.n) s = fmaf(terms.f[u], terms.y[u][at + i], s);
    if (bias) s += bias[i];
    row[i] = s;
    ss = fmaf(s, s, ss);
  }
  const float inv = 1.f / sqrtf(asb::block_sum(ss, scratch) / (float)width + eps);
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float s = row[i];
    if (out32) out32[at + i] = s;
    const float n = s * inv;
    if (out1) out1[at + i] = asb::from_float<T>(n * gain1[i]);
    if (out2) out2[at + i] = asb::from_float<T>(n * gain2[i]);
  }
}

__device__ __forceinline__ void store4(float* at, float4 v) { *reinterpret_cast<float4*>(at) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* at, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(at) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

// The same where rows are whole vectors of four: a thread keeps its NV vectors in registers, all loads of a
// term in flight together.
template <typename T, int NV>
__global__ void __launch_bounds__(256)
residual_terms_norm_vec_kernel(float* __restrict__ out32, T* __restrict__ out1, T* __restrict__ out2, const float* __restrict__ x,
                               const Terms terms, const float* __restrict__ bias, const float* __restrict__ gain1,
                               const float* __restrict__ gain2, int width, float eps) {
  __shared__ float scratch[32];
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const size_t at = (size_t)blockIdx.x * width;
  float4 s[NV];
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = (threadIdx.x + v * blockDim.x) * 4;
    s[v] = (x && i < width) ? *reinterpret_cast<const float4*>(x + at + i) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int u = 0; u < kMaxTerms; ++u) {
    if (u >= terms.n) break;
    const float f = terms.f[u];
    float4 y[NV];
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int i = (threadIdx.x + v * blockDim.x) * 4;
      y[v] = i < width ? *reinterpret_cast<const float4*>(terms.y[u] + at + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      s[v].x = fmaf(f, y[v].x, s[v].x); s[v].y = fmaf(f, y[v].y, s[v].y);
      s[v].z = fmaf(f, y[v].z, s[v].z); s[v].w = fmaf(f, y[v].w, s[v].w);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = (threadIdx.x + v * blockDim.x) * 4;
    if (bias && i < width) {
      const float4 b = *reinterpret_cast<const float4*>(bias + i);
      s[v].x += b.x; s[v].y += b.y; s[v].z += b.z; s[v].w += b.w;
    }
    ss = fmaf(s[v].x, s[v].x, fmaf(s[v].y, s[v].y, fmaf(s[v].z, s[v].z, fmaf(s[v].w, s[v].w, ss))));
  }
  float inv = 0.f;
  if (out1 || out2) inv = 1.f / sqrtf(asb::block_sum(ss, scratch) / (float)width + eps);
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int i = (threadIdx.x + v * blockDim.x) * 4;
    if (i >= width) break;
    if (out32) store4(out32 + at + i, s[v]);
    const float4 n = make_float4(s[v].x * inv, s[v].y * inv, s[v].z * inv, s[v].w * inv);
    if (out1) {
      const float4 g = *reinterpret_cast<const float4*>(gain1 + i);
      store4(out1 + at + i, make_float4(n.x * g.x, n.y * g.y, n.z * g.z, n.w * g.w));
    }
    if (out2) {
      const float4 g = *reinterpret_cast<const float4*>(gain2 + i);
      store4(out2 + at + i, make_float4(n.x * g.x, n.y * g.y, n.z * g.z, n.w * g.w));
    }
  }
}

__global__ void partial_residual_terms_norm_kernel(float* __restrict__ out32, __nv_bfloat16* __restrict__ out1,
                                                   __nv_bfloat16* __restrict__ out2, const asb::PartialSums ps, float pf,
                                                   const float* __restrict__ x, const Terms terms, const float* __restrict__ gain1,
                                                   const float* __restrict__ gain2, int width, float eps) {
  __shared__ float scratch[32];
  const int t = blockIdx.x, i = threadIdx.x * 8;
  const bool active = i < width;
  const int slots = active ? asb::partial_slots(ps, i / asb::kPartialRows) : 0;
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const size_t at = (size_t)t * width + i;
  float s[8], y[8];
#pragma unroll
  for (int k = 0; k < 8; ++k) s[k] = y[k] = 0.f;
  if (active) {
    if (x) {
      *reinterpret_cast<float4*>(s) = *reinterpret_cast<const float4*>(x + at);
      *reinterpret_cast<float4*>(s + 4) = *reinterpret_cast<const float4*>(x + at + 4);
    }
#pragma unroll
    for (int u = 0; u < kMaxTerms; ++u) {
      if (u >= terms.n) break;
      float v[8];
      *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(terms.y[u] + at);
      *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(terms.y[u] + at + 4);
#pragma unroll
      for (int k = 0; k < 8; ++k) s[k] = fmaf(terms.f[u], v[k], s[k]);
    }
    asb::partial_sum<8>(ps, t, i, slots, y);
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < 8; ++k) {
    s[k] = fmaf(pf, y[k], s[k]);
    ss = fmaf(s[k], s[k], ss);
  }
  if (active) {
    store4(out32 + at, make_float4(s[0], s[1], s[2], s[3]));
    store4(out32 + at + 4, make_float4(s[4], s[5], s[6], s[7]));
  }
  if (!out1 && !out2) return;
  const float inv = 1.f / sqrtf(asb::block_sum(ss, scratch) / (float)width + eps);
  if (!active) return;
#pragma unroll
  for (int which = 0; which < 2; ++which) {
    __nv_bfloat16* out = which ? out2 : out1;
    const float* gain = which ? gain2 : gain1;
    if (!out) continue;
#pragma unroll
    for (int k = 0; k < 8; k += 4) {
      const float4 g = *reinterpret_cast<const float4*>(gain + i + k);
      store4(out + at + k, make_float4(s[k] * inv * g.x, s[k + 1] * inv * g.y, s[k + 2] * inv * g.z, s[k + 3] * inv * g.w));
    }
  }
}

// One block per token. The block of a request's first token of the step reads the request's
// state (the id before it, plus one) and is the only one to write it (the request's last id of
// the step, plus one); every other token's predecessor is its neighbour in the flat batch.
template <typename T>
__global__ void pair_embedding_kernel(float* __restrict__ out, const T* __restrict__ table, const T* __restrict__ pairs,
                                      const int* __restrict__ ids, const int* __restrict__ positions,
                                      const int* __restrict__ req_q_start, const int* __restrict__ state_slots,
                                      int* __restrict__ last_id, int R, int width, int vocab, int buckets,
                                      int mul_prev, int mul_cur, int* __restrict__ status) {
  __shared__ int prev_s;
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const int t = blockIdx.x;
  if (threadIdx.x == 0) {
    int lo = 0, hi = R;  // the request r with req_q_start[r] <= t < req_q_start[r + 1]
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (req_q_start[mid] <= t) lo = mid; else hi = mid;
    }
    int prev;
    if (req_q_start[lo] == t) {
      const int slot = state_slots[lo];
      prev = last_id[slot] - 1;
      last_id[slot] = ids[req_q_start[lo + 1] - 1] + 1;
    } else {
      prev = ids[t - 1];
    }
    prev_s = positions[t] == 0 ? -1 : prev;
  }
  __syncthreads();
  const int id = ids[t], prev = prev_s;
  float* dst = out + (size_t)t * width;
  if (id < 0 || id >= vocab || prev >= vocab) {  // refuse rather than read outside the table
    if (threadIdx.x == 0) atomicExch(status, 1);
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = 0.f;
    return;
  }
  const long long hashed = ((long long)prev * mul_prev + (long long)id * mul_cur) % buckets;
  const T* a = table + (size_t)id * width;
  const T* b = pairs + (size_t)(prev < 0 ? buckets : (int)hashed) * width;
  if (sizeof(T) == 2 && width % 8 == 0 && (((uintptr_t)table | (uintptr_t)pairs | (uintptr_t)out) & 15) == 0) {
    // eight entries a thread: one 16-byte load from each table, two 16-byte stores
    for (int i = threadIdx.x * 8; i < width; i += blockDim.x * 8) {
      const uint4 ra = *reinterpret_cast<const uint4*>(a + i), rb = *reinterpret_cast<const uint4*>(b + i);
      const __nv_bfloat162* ha = reinterpret_cast<const __nv_bfloat162*>(&ra);
      const __nv_bfloat162* hb = reinterpret_cast<const __nv_bfloat162*>(&rb);
      float sum[8];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float2 fa = __bfloat1622float2(ha[u]), fb = __bfloat1622float2(hb[u]);
        sum[2 * u] = fa.x + fb.x;
        sum[2 * u + 1] = fa.y + fb.y;
      }
      *reinterpret_cast<float4*>(dst + i) = make_float4(sum[0], sum[1], sum[2], sum[3]);
      *reinterpret_cast<float4*>(dst + i + 4) = make_float4(sum[4], sum[5], sum[6], sum[7]);
    }
    return;
  }
  for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = asb::to_float(a[i]) + asb::to_float(b[i]);
}

template <typename T>
__global__ void concat_cast_kernel(T* __restrict__ out, const float* __restrict__ a, const float* __restrict__ b,
                                   int width, long long total) {
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  if (width % 4 == 0 && (((uintptr_t)a | (uintptr_t)b | (uintptr_t)out) & 15) == 0) {
    // four entries a thread (no group of four straddles the two halves of a row)
    for (long long i = (blockIdx.x * (long long)blockDim.x + threadIdx.x) * 4; i < total; i += (long long)gridDim.x * blockDim.x * 4) {
      const long long r = i / (2 * width);
      const int c = (int)(i - r * 2 * width);
      const float4 v = *reinterpret_cast<const float4*>(c < width ? a + r * width + c : b + r * width + c - width);
      if (sizeof(T) == 2) {  // one 8-byte store
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
        *reinterpret_cast<uint2*>(out + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
      } else {
        out[i] = asb::from_float<T>(v.x);
        out[i + 1] = asb::from_float<T>(v.y);
        out[i + 2] = asb::from_float<T>(v.z);
        out[i + 3] = asb::from_float<T>(v.w);
      }
    }
    return;
  }
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / (2 * width);
    const int c = (int)(i - r * 2 * width);
    out[i] = asb::from_float<T>(c < width ? a[r * width + c] : b[r * width + c - width]);
  }
}

}  // namespace

// out32, out1, out2, x, bias: each may be null (out1 with gain1, out2 with gain2); y1 .. y4 with their factors:
// the first `terms` of them. dtype is that of out1 and out2.
extern "C" int asb_residual_terms_norm(float* out32, void* out1, void* out2, const float* x, const float* y1, const float* y2,
                                       const float* y3, const float* y4, float f1, float f2, float f3, float f4, int terms,
                                       const float* bias, const float* gain1, const float* gain2, int n, int width, float eps,
                                       int dtype, cudaStream_t stream) {
  if (n == 0) return 0;
  if (width < 1 || width > 48 * 1024 / 4) return asb::fail("residual_terms_norm: width %d not in 1..12288", width);
  if (terms < 0 || terms > kMaxTerms) return asb::fail("residual_terms_norm: %d terms, at most %d", terms, kMaxTerms);
  if ((out1 && !gain1) || (out2 && !gain2)) return asb::fail("residual_terms_norm: a normed output needs its gain");
  const Terms t = {{y1, y2, y3, y4}, {f1, f2, f3, f4}, terms};
  uintptr_t all = (uintptr_t)out32 | (uintptr_t)out1 | (uintptr_t)out2 | (uintptr_t)x | (uintptr_t)bias | (uintptr_t)gain1 | (uintptr_t)gain2;
  for (int u = 0; u < terms; ++u) {
    if (!t.y[u]) return asb::fail("residual_terms_norm: term %d is missing", u);
    all |= (uintptr_t)t.y[u];
  }
  if (width % 4 == 0 && width <= 8192 && (all & 15) == 0) {
    const int vectors = width / 4, nv = vectors <= 256 ? 1 : (vectors <= 512 ? 2 : (vectors <= 1024 ? 4 : 8));
    const int threads = ((vectors + nv - 1) / nv + 31) / 32 * 32;
#define ASB_TERMS(NV)                                                                                                     \
  ASB_DISPATCH_DTYPE(dtype, T, asb::launch(residual_terms_norm_vec_kernel<T, NV>, n, threads, 0, stream, out32, (T*)out1, \
                                           (T*)out2, x, t, bias, gain1, gain2, width, eps))
    if (nv == 1) ASB_TERMS(1);
    else if (nv == 2) ASB_TERMS(2);
    else if (nv == 4) ASB_TERMS(4);
    else ASB_TERMS(8);
#undef ASB_TERMS
    return asb::check_launch("residual_terms_norm");
  }
  ASB_DISPATCH_DTYPE(dtype, T, asb::launch(residual_terms_norm_kernel<T>, n, threads_for(width), width * sizeof(float),
                                           stream, out32, (T*)out1, (T*)out2, x, t, bias, gain1, gain2, width, eps));
  return asb::check_launch("residual_terms_norm");
}

// The form with a last term f y given as partial sums (asb_gemm_tcgen05 mode 3 on [n, K] x [width, K]); out1 and
// out2 are bfloat16. Widths that are a multiple of 8 up to 8192, pointers 16-byte aligned.
extern "C" int asb_partial_residual_terms_norm(float* out32, void* out1, void* out2, const float* ws, int max_slots, int bn,
                                               int kb_per_tile, int num_tiles, int blocks, float f, const float* x, const float* y1,
                                               const float* y2, const float* y3, const float* y4, float f1, float f2, float f3,
                                               float f4, int terms, const float* gain1, const float* gain2, int n, int width,
                                               float eps, cudaStream_t stream) {
  if (n == 0) return 0;
  if (width % 8 || width / 8 > 1024) return asb::fail("partial_residual_terms_norm: width %d must be a multiple of 8 up to 8192", width);
  if (n > bn || num_tiles * asb::kPartialRows < width)
    return asb::fail("partial_residual_terms_norm: %d tokens x %d columns do not fit the partial sums (%d x %d)", n, width, bn,
                     num_tiles * asb::kPartialRows);
  if (terms < 0 || terms > kMaxTerms) return asb::fail("partial_residual_terms_norm: %d terms, at most %d", terms, kMaxTerms);
  if (!out32 || (out1 && !gain1) || (out2 && !gain2)) return asb::fail("partial_residual_terms_norm: outputs and their gains");
  const Terms t = {{y1, y2, y3, y4}, {f1, f2, f3, f4}, terms};
  uintptr_t all = (uintptr_t)out32 | (uintptr_t)out1 | (uintptr_t)out2 | (uintptr_t)x | (uintptr_t)gain1 | (uintptr_t)gain2 | (uintptr_t)ws;
  for (int u = 0; u < terms; ++u) {
    if (!t.y[u]) return asb::fail("partial_residual_terms_norm: term %d is missing", u);
    all |= (uintptr_t)t.y[u];
  }
  if (all & 15) return asb::fail("partial_residual_terms_norm: pointers must be 16-byte aligned");
  const asb::PartialSums ps = {ws, max_slots, bn, kb_per_tile, num_tiles, blocks};
  asb::launch(partial_residual_terms_norm_kernel, n, ((width / 8) + 31) / 32 * 32, 0, stream, out32, (__nv_bfloat16*)out1,
              (__nv_bfloat16*)out2, ps, f, x, t, gain1, gain2, width, eps);
  return asb::check_launch("partial_residual_terms_norm");
}

extern "C" int asb_pair_embedding(float* out, const void* table, const void* pairs, const int* ids,
                                  const int* positions, const int* req_q_start, const int* state_slots,
                                  int* last_id, int num_tokens, int R, int width, int vocab, int buckets,
                                  int mul_prev, int mul_cur, int dtype, int* status, cudaStream_t stream) {
  if (num_tokens == 0) return 0;
  if (buckets < 1 || R < 1) return asb::fail("pair_embedding: %d buckets, %d requests", buckets, R);
  ASB_DISPATCH_DTYPE(dtype, T, asb::launch(pair_embedding_kernel<T>, num_tokens, threads_for(sizeof(T) == 2 && width % 8 == 0 ? width / 8 : width), 0, stream, out,
                                           (const T*)table, (const T*)pairs, ids, positions, req_q_start, state_slots,
                                           last_id, R, width, vocab, buckets, mul_prev, mul_cur, status));
  return asb::check_launch("pair_embedding");
}

extern "C" int asb_concat_cast(void* out, const float* a, const float* b, int n, int width, int dtype,
                               cudaStream_t stream) {
  if (n == 0) return 0;
  const long long total = (long long)n * 2 * width;
  const long long blocks = (total / (width % 4 == 0 ? 4 : 1) + 255) / 256;
  ASB_DISPATCH_DTYPE(dtype, T, asb::launch(concat_cast_kernel<T>, (unsigned)(blocks < 148 * 16 ? blocks : 148 * 16), 256,
                                           0, stream, (T*)out, a, b, width, total));
  return asb::check_launch("concat_cast");
}
