// Kernels for blocks over several parallel residual streams ("hyper-connections"): S float32 copies
// x_1 .. x_S of the residual per token. A sublayer f reads a weighted sum of them and its output goes
// back to all of them while they are mixed with one another:
//
//   u = sum_s in[s] x_s;   y = f(N(u));   x_t <- sum_s mix[s, t] x_s + out[t] y
//
//   asb_hyper_streams   one pass over a token's streams that closes one sublayer and opens the next:
//                       the new streams from the old ones and y (+ a bias), written as float32, and
//                       N(sum_s in[s] x_s) * gain in the compute dtype, in and gain those of
//                       whatever reads the streams next; N is the centred norm
//                       (u - mean) / sqrt(var + eps) or the RMS norm. Either half may be absent
//                       (a model's first sublayer only reads; its last only writes), rows may be
//                       gathered (the final norm of the rows whose logits are wanted), and the
//                       streams may be read with a stream stride of 0: S copies of one row.
//
// y comes as float32 rows, as the partial sums that the tensor-core GEMM left in its workspace (few
// tokens), or as the routed experts' output rows with each token's choices and weights: the kernel
// then adds them up itself. Everything is float32; each stored value is rounded once.
#include "common.cuh"
#include "gemm_partials.cuh"

namespace {

constexpr int kMaxStreams = 16;
enum Source : int { kNone = 0, kRows = 1, kPartial = 2, kExperts = 3 };

struct HyperParams {
  float* out;         // [n, S, width] or null
  void* normed;       // [n, width] in the compute dtype, or null
  const float* x;     // stream s of token t at x + t * token_stride + s * stream_stride
  long long token_stride, stream_stride;
  const int* rows;    // [n] source tokens, or null
  const float* y;     // kRows: [n, width]; kExperts: the sorted rows' outputs [pairs, width]
  const int* pair_row;   // kExperts: [n, top]
  const float* pair_weight;
  int top;
  asb::PartialSums ps;   // kPartial
  const float* bias;  // [width] or null
  const float* w_out; // [S]
  const float* w_mix; // [S, S], [from, to]
  const float* w_in;  // [S]
  const float* gain;  // [width]
  int S, width, source, centred;
  float eps;
};

template <int V>
__device__ __forceinline__ void load_v(float (&v)[V], const float* at) {
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(at);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    v[0] = *at;
  }
}
template <int V>
__device__ __forceinline__ void store_v(float* at, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(at) = make_float4(v[0], v[1], v[2], v[3]);
  else *at = v[0];
}
template <typename T, int V>
__device__ __forceinline__ void store_c(T* at, const float (&v)[V]) {
  if constexpr (sizeof(T) == 4) {
    store_v<V>((float*)at, v);
  } else if constexpr (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(at) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
  } else {
    *at = asb::from_float<T>(v[0]);
  }
}

// the sublayer's output, V columns from i on, of output row t
template <int V>
__device__ __forceinline__ void sublayer_output(const HyperParams& p, int t, int i, float (&y)[V]) {
#pragma unroll
  for (int k = 0; k < V; ++k) y[k] = 0.f;
  if (p.source == kRows) {
    load_v<V>(y, p.y + (size_t)t * p.width + i);
  } else if (p.source == kPartial) {
    asb::partial_sum<V>(p.ps, t, i, asb::partial_slots(p.ps, i / asb::kPartialRows), y);
  } else if (p.source == kExperts) {
    for (int c = 0; c < p.top; ++c) {  // the choices in their order of selection
      const size_t pair = (size_t)t * p.top + c;
      const float w = p.pair_weight[pair];
      float v[V];
      load_v<V>(v, p.y + (size_t)p.pair_row[pair] * p.width + i);
#pragma unroll
      for (int k = 0; k < V; ++k) y[k] = fmaf(w, v[k], y[k]);
    }
  }
  if (p.bias) {
    float b[V];
    load_v<V>(b, p.bias + i);
#pragma unroll
    for (int k = 0; k < V; ++k) y[k] += b[k];
  }
}

// One block per output row; S = 0: any number of streams, read again for every new one (the streams
// are written to another buffer than they are read from).
template <typename T, int S, int V>
__global__ void __launch_bounds__(1024)
hyper_streams_kernel(const HyperParams p) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[32];
  __shared__ float mix[kMaxStreams * kMaxStreams], out_w[kMaxStreams], in_w[kMaxStreams];
  const int n_streams = S > 0 ? S : p.S;
  for (int i = threadIdx.x; i < n_streams * n_streams; i += blockDim.x) mix[i] = p.w_mix ? p.w_mix[i] : 0.f;
  for (int i = threadIdx.x; i < n_streams; i += blockDim.x) {
    out_w[i] = p.w_out ? p.w_out[i] : 0.f;
    in_w[i] = p.w_in ? p.w_in[i] : 0.f;
  }
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  __syncthreads();
  const int t = blockIdx.x, width = p.width;
  const size_t src = p.rows ? (size_t)p.rows[t] : (size_t)t;
  const float* x = p.x + src * p.token_stride;
  float* out = p.out ? p.out + (size_t)t * n_streams * width : nullptr;
  const bool advance = p.w_mix != nullptr;
  float sum = 0.f;
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    float y[V], u[V];
    sublayer_output<V>(p, t, i, y);
#pragma unroll
    for (int k = 0; k < V; ++k) u[k] = 0.f;
    if constexpr (S > 0) {
      float v[S][V];
#pragma unroll
      for (int s = 0; s < S; ++s) load_v<V>(v[s], x + s * p.stream_stride + i);
#pragma unroll
      for (int to = 0; to < S; ++to) {
        float nv[V];
        if (advance) {
#pragma unroll
          for (int k = 0; k < V; ++k) nv[k] = out_w[to] * y[k];
#pragma unroll
          for (int s = 0; s < S; ++s)
#pragma unroll
            for (int k = 0; k < V; ++k) nv[k] = fmaf(mix[s * S + to], v[s][k], nv[k]);
        } else {
#pragma unroll
          for (int k = 0; k < V; ++k) nv[k] = v[to][k];
        }
        if (out) store_v<V>(out + (size_t)to * width + i, nv);
#pragma unroll
        for (int k = 0; k < V; ++k) u[k] = fmaf(in_w[to], nv[k], u[k]);
      }
    } else {
      for (int to = 0; to < n_streams; ++to) {
        float nv[V], v[V];
        if (advance) {
#pragma unroll
          for (int k = 0; k < V; ++k) nv[k] = out_w[to] * y[k];
          for (int s = 0; s < n_streams; ++s) {
            load_v<V>(v, x + s * p.stream_stride + i);
#pragma unroll
            for (int k = 0; k < V; ++k) nv[k] = fmaf(mix[s * n_streams + to], v[k], nv[k]);
          }
        } else {
          load_v<V>(nv, x + to * p.stream_stride + i);
        }
        if (out) store_v<V>(out + (size_t)to * width + i, nv);
#pragma unroll
        for (int k = 0; k < V; ++k) u[k] = fmaf(in_w[to], nv[k], u[k]);
      }
    }
    store_v<V>(row + i, u);  // (each thread reads back only what it wrote itself)
#pragma unroll
    for (int k = 0; k < V; ++k) sum += u[k];
  }
  if (!p.normed) return;
  const float inv_w = 1.f / (float)width;
  const float mean = p.centred ? asb::block_sum(sum, scratch) * inv_w : 0.f;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    float u[V];
    load_v<V>(u, row + i);
#pragma unroll
    for (int k = 0; k < V; ++k) ss = fmaf(u[k] - mean, u[k] - mean, ss);
  }
  const float inv = 1.f / sqrtf(asb::block_sum(ss, scratch) * inv_w + p.eps);
  T* normed = (T*)p.normed + (size_t)t * width;
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    float u[V], g[V];
    load_v<V>(u, row + i);
    load_v<V>(g, p.gain + i);
#pragma unroll
    for (int k = 0; k < V; ++k) u[k] = (u[k] - mean) * inv * g[k];
    store_c<T, V>(normed + i, u);
  }
}

template <typename T, int S, int V>
int run(const HyperParams& p, int n, cudaStream_t stream) {
  const size_t smem = sizeof(float) * (size_t)p.width;
  auto kern = hyper_streams_kernel<T, S, V>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return asb::fail("hyper_streams: width %d: %s", p.width, cudaGetErrorString(e));
  }
  // few rows: as many threads as a row has vectors; many rows: blocks of up to 512, several to an SM
  const int vectors = (p.width + V - 1) / V, most = n <= 296 ? 1024 : 512;
  int threads = 64;
  while (threads < vectors && threads < most) threads <<= 1;
  asb::launch(kern, n, threads, smem, stream, p);
  return asb::check_launch("hyper_streams");
}

template <typename T>
int dispatch(const HyperParams& p, int n, cudaStream_t stream) {
  const bool wide = p.width % 4 == 0 && p.token_stride % 4 == 0 && p.stream_stride % 4 == 0 &&
                    (((uintptr_t)p.out | (uintptr_t)p.normed | (uintptr_t)p.x | (uintptr_t)p.y | (uintptr_t)p.ps.ws |
                      (uintptr_t)p.bias | (uintptr_t)p.gain) & 15) == 0;
  if (!wide) return run<T, 0, 1>(p, n, stream);
  switch (p.S) {
    case 1: return run<T, 1, 4>(p, n, stream);
    case 2: return run<T, 2, 4>(p, n, stream);
    case 3: return run<T, 3, 4>(p, n, stream);
    case 4: return run<T, 4, 4>(p, n, stream);
    default: return run<T, 0, 4>(p, n, stream);
  }
}

}  // namespace

// source 0: no sublayer output (then w_out and w_mix are null and the streams are only read); 1: y
// float32 [n, width]; 2: partial sums of asb_gemm_tcgen05 mode 3 (ws and the five numbers of its
// layout); 3: y the experts' rows, pair_row and pair_weight [n, top]. out, normed (with gain and
// w_in), rows, bias: each may be null. dtype is that of `normed`.
extern "C" int asb_hyper_streams(float* out, void* normed, const float* x, long long token_stride, long long stream_stride,
                                 const int* rows, int source, const float* y, const int* pair_row,
                                 const float* pair_weight, int top, const float* ws, int max_slots, int bn,
                                 int kb_per_tile, int num_tiles, int blocks, const float* bias, const float* w_out,
                                 const float* w_mix, const float* w_in, const float* gain, int n, int S, int width,
                                 float eps, int centred, int dtype, cudaStream_t stream) {
  if (n == 0) return 0;
  if (S < 1 || S > kMaxStreams) return asb::fail("hyper_streams: %d streams, at most %d", S, kMaxStreams);
  if (width < 1 || (size_t)width * 4 > 200 * 1024) return asb::fail("hyper_streams: width %d", width);
  if (source < kNone || source > kExperts || (source != kNone) != (w_mix != nullptr) || (w_mix && !w_out))
    return asb::fail("hyper_streams: a sublayer's output needs the streams' weights, and the other way round");
  if ((source == kRows && !y) || (source == kExperts && (!y || !pair_row || !pair_weight || top < 1)))
    return asb::fail("hyper_streams: source %d lacks its rows", source);
  if (source == kPartial && (!ws || n > bn || num_tiles * asb::kPartialRows < width))
    return asb::fail("hyper_streams: %d rows x %d columns do not fit the partial sums", n, width);
  if (normed && (!gain || !w_in)) return asb::fail("hyper_streams: a normed output needs its gain and the streams' input weights");
  if (rows && w_mix) return asb::fail("hyper_streams: rows are gathered for reading only");
  HyperParams p;
  p.out = out; p.normed = normed; p.x = x; p.token_stride = token_stride; p.stream_stride = stream_stride;
  p.rows = rows; p.y = y; p.pair_row = pair_row; p.pair_weight = pair_weight; p.top = top;
  p.ps = asb::PartialSums{ws, max_slots, bn, kb_per_tile, num_tiles, blocks};
  p.bias = bias; p.w_out = w_out; p.w_mix = w_mix; p.w_in = w_in; p.gain = gain;
  p.S = S; p.width = width; p.source = source; p.centred = centred; p.eps = eps;
  ASB_DISPATCH_DTYPE(dtype, T, return dispatch<T>(p, n, stream));
  return 0;
}
