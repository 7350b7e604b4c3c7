// The gated delta rule, a recurrence over a request's tokens with a matrix state per head:
//
//   S <- g_t S;  u_t = beta_t (v_t - S^T k_t);  S <- S + k_t u_t^T;  o_t = S^T q_t
//
// S: [D, V] per (request, head), float32, kept in the request's state slot between steps. q and k are
// made unit vectors per head (x / sqrt(sum x^2 + 1e-6)), q times D^(-1/2) besides; neighbouring heads
// may share one q and one k. Per head beta = sigmoid(zb) and g = exp(-exp(A) softplus(za + dt_bias)).
// q, k and v are column ranges of one tensor [T, stride] in the compute dtype (the short convolutions'
// output); everything from there on is float32: unit norms, gates, state, products, outputs.
//
// Two forms of the same sums:
//
//   asb_delta_step    token by token, for single tokens and short portions. With a = S^T k and
//                     b = S^T q of the state before the token, u = beta (v - g a),
//                     o = g b + (k . q) u and S <- g S + k u^T, so a token reads the state once. A block
//                     owns (request, head, slice of value columns): each of its 8 warps holds a share
//                     of the rows in registers (a lane 1, 2 or 4 neighbouring columns), and the warps'
//                     parts of a and b meet in shared memory, one barrier a token.
//
//   asb_delta_chunks  long portions, in chunks of C tokens. With G_i the sum of log g up to token i of
//                     the chunk, all u of a chunk solve a unit lower triangular system,
//                       (I + L) U = diag(beta) (V - diag(e^G) K S),  L_ij = beta_i e^(G_i - G_j) k_i . k_j (j < i),
//                     so with Y = (I + L)^-1 diag(beta) V and W = (I + L)^-1 diag(beta e^G) K
//                       U = Y - W S,   O = diag(e^G) Q S + P U,  P_ij = e^(G_i - G_j) q_i . k_j (j <= i),
//                       S <- e^(G_C) S + (diag(e^(G_C - G)) K)^T U.
//                     The first kernel (a block per chunk and head, all at once) makes Y, W, P and the
//                     scaled Q and K; the second walks a request's chunks in order, a block per
//                     (request, head, slice of value columns) with its slice of S in shared memory,
//                     four small matrix products a chunk on float32 multiply-adds, the next chunk's
//                     operands arriving while this one's are multiplied.
//
// Chunks are counted from a step's first token, so where a prompt is cut only regroups sums.
#include "attention_mma.cuh"

namespace {

using asb::mma::cp_async16;
using asb::mma::cp_async_commit;
using asb::mma::cp_async_wait;
using asb::mma::smem_u32;

constexpr float kUnitEps = 1e-6f;

struct DeltaInputs {
  const void* x;           // [T, stride]: q [G][D] from q_off, k [G][D] from k_off, v [H][V] from v_off
  const float* z;          // [T, z_stride]: beta's pre-activations [H] from b_off, the decay's [H] from a_off
  const float* dt_bias;    // [H]
  const float* a_log;      // [H]
  int stride, q_off, k_off, v_off, z_stride, b_off, a_off;
  int H, D, V, share;      // share: heads that read one q and one k
  float q_scale;
};

struct StepParams {
  DeltaInputs in;
  float* out;              // [T, H * V]
  float* state;            // [slots, H, D, V]
  const int* state_slots;  // [R]
  const int* req_q_start;  // [R + 1]
  int limit;               // requests bringing more tokens are left to asb_delta_chunks; 0: none are
};

__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float log_decay(const DeltaInputs& in, size_t row, int h) {
  return -expf(in.a_log[h]) * softplus_f(in.z[row * in.z_stride + in.a_off + h] + in.dt_bias[h]);
}
__device__ __forceinline__ float beta_of(const DeltaInputs& in, size_t row, int h) {
  return 1.f / (1.f + expf(-in.z[row * in.z_stride + in.b_off + h]));
}

// One warp: token `row`'s unit vectors of head h into q_s and k_s (zeros from D to `padded`); q . k in every lane.
template <typename T>
__device__ __forceinline__ float unit_qk(const DeltaInputs& in, size_t row, int h, float* q_s, float* k_s, int padded, int lane) {
  const T* at = (const T*)in.x + row * in.stride + (h / in.share) * in.D;
  float qq = 0.f, kk = 0.f, qk = 0.f;
  for (int d = lane; d < padded; d += 32) {
    const bool in_row = d < in.D;
    const float q = in_row ? asb::to_float(at[in.q_off + d]) : 0.f, k = in_row ? asb::to_float(at[in.k_off + d]) : 0.f;
    q_s[d] = q;
    k_s[d] = k;
    qq = fmaf(q, q, qq);
    kk = fmaf(k, k, kk);
    qk = fmaf(q, k, qk);
  }
  const float rq = in.q_scale / sqrtf(asb::warp_sum(qq) + kUnitEps), rk = 1.f / sqrtf(asb::warp_sum(kk) + kUnitEps);
  for (int d = lane; d < padded; d += 32) {  // (each lane rescales what it wrote)
    q_s[d] *= rq;
    k_s[d] *= rk;
  }
  return asb::warp_sum(qk) * rq * rk;
}

// ---- token by token -------------------------------------------------------------------------

constexpr int kStepWarps = 8;

template <int CV> struct Columns;
template <> struct Columns<1> {
  static __device__ __forceinline__ void load(const float* at, float* v) { v[0] = at[0]; }
  static __device__ __forceinline__ void store(float* at, const float* v) { at[0] = v[0]; }
};
template <> struct Columns<2> {
  static __device__ __forceinline__ void load(const float* at, float* v) {
    const float2 f = *reinterpret_cast<const float2*>(at);
    v[0] = f.x; v[1] = f.y;
  }
  static __device__ __forceinline__ void store(float* at, const float* v) { *reinterpret_cast<float2*>(at) = make_float2(v[0], v[1]); }
};
template <> struct Columns<4> {
  static __device__ __forceinline__ void load(const float* at, float* v) {
    const float4 f = *reinterpret_cast<const float4*>(at);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  }
  static __device__ __forceinline__ void store(float* at, const float* v) {
    *reinterpret_cast<float4*>(at) = make_float4(v[0], v[1], v[2], v[3]);
  }
};

// RPT: rows of S a warp holds (8 * RPT >= D); CV: neighbouring columns a lane owns (V a multiple of it).
template <typename T, int RPT, int CV>
__global__ void __launch_bounds__(kStepWarps * 32)
delta_step_kernel(const StepParams p) {
  constexpr int DP = kStepWarps * RPT, VS = 32 * CV;
  extern __shared__ __align__(16) float smem[];
  float* qs = smem;                      // [8][DP], a token per warp
  float* ks = qs + kStepWarps * DP;      // [8][DP]
  float* vs = ks + kStepWarps * DP;      // [8][VS]
  float* part = vs + kStepWarps * VS;    // [2][2][8][VS]: the warps' shares of a and of b, for two tokens in turn
  __shared__ float g_s[kStepWarps], beta_s[kStepWarps], kq_s[kStepWarps];
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const DeltaInputs& in = p.in;
  const int r = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row_lo = p.req_q_start[r], row_hi = p.req_q_start[r + 1];
  if (row_hi == row_lo || (p.limit > 0 && row_hi - row_lo > p.limit)) return;
  const int col = blockIdx.z * VS + lane * CV;
  const bool live = col < in.V;
  float* sp = p.state + (((size_t)p.state_slots[r] * in.H + h) * in.D) * in.V + col;
  float S[RPT][CV];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = warp * RPT + i;
    if (live && d < in.D) {
      Columns<CV>::load(sp + (size_t)d * in.V, S[i]);
    } else {
#pragma unroll
      for (int c = 0; c < CV; ++c) S[i][c] = 0.f;
    }
  }
  for (int t0 = row_lo; t0 < row_hi; t0 += kStepWarps) {
    const int nt = min(kStepWarps, row_hi - t0);
    if (t0 != row_lo) __syncthreads();  // the last tile's vectors have been read
    if (warp < nt) {
      const size_t row = (size_t)(t0 + warp);
      const T* vrow = (const T*)in.x + row * in.stride + in.v_off + h * in.V;
#pragma unroll
      for (int c = 0; c < CV; ++c) vs[warp * VS + lane * CV + c] = live ? asb::to_float(vrow[col + c]) : 0.f;
      const float kq = unit_qk<T>(in, row, h, qs + warp * DP, ks + warp * DP, DP, lane);
      if (lane == 0) {
        g_s[warp] = expf(log_decay(in, row, h));
        beta_s[warp] = beta_of(in, row, h);
        kq_s[warp] = kq;
      }
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float* qr = qs + t * DP + warp * RPT;
      const float* kr = ks + t * DP + warp * RPT;
      float a[CV], b[CV];
#pragma unroll
      for (int c = 0; c < CV; ++c) a[c] = b[c] = 0.f;
#pragma unroll
      for (int i = 0; i < RPT; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(kr + i), q4 = *reinterpret_cast<const float4*>(qr + i);
        const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int c = 0; c < CV; ++c) {
            a[c] = fmaf(S[i + j][c], kk[j], a[c]);
            b[c] = fmaf(S[i + j][c], qq[j], b[c]);
          }
      }
      float* pa = part + (t & 1) * 2 * kStepWarps * VS;
      float* pb = pa + kStepWarps * VS;
      Columns<CV>::store(pa + warp * VS + lane * CV, a);
      Columns<CV>::store(pb + warp * VS + lane * CV, b);
      __syncthreads();
      const float g = g_s[t], beta = beta_s[t];
      float u[CV];
#pragma unroll
      for (int c = 0; c < CV; ++c) u[c] = 0.f;
#pragma unroll
      for (int w = 0; w < kStepWarps; ++w) {
        float v[CV];
        Columns<CV>::load(pa + w * VS + lane * CV, v);
#pragma unroll
        for (int c = 0; c < CV; ++c) u[c] += v[c];
      }
#pragma unroll
      for (int c = 0; c < CV; ++c) u[c] = beta * fmaf(-g, u[c], vs[t * VS + lane * CV + c]);
      if (warp == t && live) {
        float o[CV];
#pragma unroll
        for (int c = 0; c < CV; ++c) o[c] = 0.f;
#pragma unroll
        for (int w = 0; w < kStepWarps; ++w) {
          float v[CV];
          Columns<CV>::load(pb + w * VS + lane * CV, v);
#pragma unroll
          for (int c = 0; c < CV; ++c) o[c] += v[c];
        }
#pragma unroll
        for (int c = 0; c < CV; ++c) o[c] = fmaf(g, o[c], kq_s[t] * u[c]);
        Columns<CV>::store(p.out + ((size_t)(t0 + t) * in.H + h) * in.V + col, o);
      }
#pragma unroll
      for (int i = 0; i < RPT; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(kr + i);
        const float kk[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int c = 0; c < CV; ++c) S[i + j][c] = fmaf(g, S[i + j][c], kk[j] * u[c]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = warp * RPT + i;
    if (live && d < in.D) Columns<CV>::store(sp + (size_t)d * in.V, S[i]);
  }
}

template <typename T, int RPT, int CV>
int launch_step(const StepParams& p, int R, cudaStream_t stream) {
  const size_t smem = sizeof(float) * kStepWarps * (2 * kStepWarps * RPT + 32 * CV + 4 * 32 * CV);
  auto kern = delta_step_kernel<T, RPT, CV>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return asb::fail("delta_step: shared memory %zu: %s", smem, cudaGetErrorString(e));
  }
  dim3 grid(R, p.in.H, (p.in.V + 32 * CV - 1) / (32 * CV));
  asb::launch(kern, grid, kStepWarps * 32, smem, stream, p);
  return asb::check_launch("delta_step");
}

template <typename T, int RPT>
int launch_step_columns(const StepParams& p, int R, int cv, cudaStream_t stream) {
  if (cv == 4) return launch_step<T, RPT, 4>(p, R, stream);
  if (cv == 2) return launch_step<T, RPT, 2>(p, R, stream);
  return launch_step<T, RPT, 1>(p, R, stream);
}

// ---- in chunks ------------------------------------------------------------------------------

constexpr int kPrepareThreads = 256;

struct ChunkParams {
  DeltaInputs in;
  float* out;              // [T, H * V]
  float* state;            // [slots, H, D, V]
  const int* state_slots;  // [R]
  const int* chunk_row;    // [chunks] first row of each chunk
  const int* chunk_len;    // [chunks] tokens, 1 .. C
  const int* req;          // [n, 3]: request, its first chunk, its chunks
  // what the first kernel leaves for the second, per (chunk, head)
  float* wq;               // [chunks, H, DP, 2 C]: per row d of S the C entries of W, then those of e^G Q
  float* kd;               // [chunks, H, C, DP]: e^(G_C - G) K
  float* pt;               // [chunks, H, C, C]: P transposed, [j][i]
  float* y;                // [chunks, H, C, VP]
  float* through;          // [chunks, H]: e^(G_C)
  int DP, VP;              // D to a multiple of 4, V to a multiple of 32
};

template <typename T, int C>
__global__ void __launch_bounds__(kPrepareThreads, 2)
delta_chunk_prepare_kernel(const ChunkParams p) {
  constexpr int TI = C / 16, LA = C + 4;
  extern __shared__ __align__(16) float smem[];
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const DeltaInputs& in = p.in;
  const int DP = p.DP, LD = DP + 4;
  float* ks = smem;             // [C][LD]
  float* qs = ks + C * LD;      // [C][LD]
  float* L = qs + C * LD;       // [C][LA]
  float* G = L + C * LA;        // [C]
  float* beta = G + C;          // [C]
  float* eg = beta + C;         // [C]
  const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row0 = p.chunk_row[chunk], n = p.chunk_len[chunk];
  const size_t at = (size_t)chunk * in.H + h;
  // rows past the chunk's tokens: zero vectors, beta 0, decay 1; they change nothing
  // (four rows a warp at a time, their loads in flight together)
  for (int i0 = warp * 4; i0 < C; i0 += kPrepareThreads / 8) {
    const T* src = (const T*)in.x + (size_t)(row0 + i0) * in.stride + (h / in.share) * in.D;
    float qq[4] = {0.f, 0.f, 0.f, 0.f}, kk[4] = {0.f, 0.f, 0.f, 0.f};
    for (int d = lane; d < DP; d += 32) {
      float q[4], k[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const bool real = i0 + u < n && d < in.D;
        q[u] = real ? asb::to_float(src[(size_t)u * in.stride + in.q_off + d]) : 0.f;
        k[u] = real ? asb::to_float(src[(size_t)u * in.stride + in.k_off + d]) : 0.f;
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        qs[(i0 + u) * LD + d] = q[u];
        ks[(i0 + u) * LD + d] = k[u];
        qq[u] = fmaf(q[u], q[u], qq[u]);
        kk[u] = fmaf(k[u], k[u], kk[u]);
      }
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1)
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        qq[u] += __shfl_xor_sync(0xffffffffu, qq[u], off);
        kk[u] += __shfl_xor_sync(0xffffffffu, kk[u], off);
      }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float rq = in.q_scale / sqrtf(qq[u] + kUnitEps), rk = 1.f / sqrtf(kk[u] + kUnitEps);
      for (int d = lane; d < DP; d += 32) {  // (each lane rescales what it wrote)
        qs[(i0 + u) * LD + d] *= rq;
        ks[(i0 + u) * LD + d] *= rk;
      }
    }
  }
  if (warp == 0) {
    float before = 0.f;
    for (int i0 = 0; i0 < C; i0 += 32) {
      const int i = i0 + lane;
      float s = i < n ? log_decay(in, (size_t)(row0 + i), h) : 0.f;
#pragma unroll
      for (int off = 1; off < 32; off <<= 1) {
        const float other = __shfl_up_sync(0xffffffffu, s, off);
        if (lane >= off) s += other;
      }
      s += before;
      before = __shfl_sync(0xffffffffu, s, 31);
      G[i] = s;
      eg[i] = expf(s);
      beta[i] = i < n ? beta_of(in, (size_t)(row0 + i), h) : 0.f;
    }
  }
  __syncthreads();
  {
    // K K^T and Q K^T: a thread owns rows ti + 16 a and columns tj + 16 b
    const int ti = tid & 15, tj = tid >> 4;
    float kk[TI][TI], qk[TI][TI];
#pragma unroll
    for (int a = 0; a < TI; ++a)
#pragma unroll
      for (int b = 0; b < TI; ++b) kk[a][b] = qk[a][b] = 0.f;
    for (int d = 0; d < DP; d += 4) {
      float4 kc[TI];
#pragma unroll
      for (int b = 0; b < TI; ++b) kc[b] = *reinterpret_cast<const float4*>(ks + (tj + 16 * b) * LD + d);
#pragma unroll
      for (int a = 0; a < TI; ++a) {
        const float4 kr = *reinterpret_cast<const float4*>(ks + (ti + 16 * a) * LD + d);
        const float4 qr = *reinterpret_cast<const float4*>(qs + (ti + 16 * a) * LD + d);
#pragma unroll
        for (int b = 0; b <= a; ++b) {  // (sub-blocks above the diagonal are not needed)
          kk[a][b] = fmaf(kr.x, kc[b].x, fmaf(kr.y, kc[b].y, fmaf(kr.z, kc[b].z, fmaf(kr.w, kc[b].w, kk[a][b]))));
          qk[a][b] = fmaf(qr.x, kc[b].x, fmaf(qr.y, kc[b].y, fmaf(qr.z, kc[b].z, fmaf(qr.w, kc[b].w, qk[a][b]))));
        }
      }
    }
    float* pt = p.pt + at * C * C;
#pragma unroll
    for (int a = 0; a < TI; ++a)
#pragma unroll
      for (int b = 0; b < TI; ++b) {
        const int i = ti + 16 * a, j = tj + 16 * b;
        if (b > a) {
          L[i * LA + j] = 0.f;
          pt[j * C + i] = 0.f;
          continue;
        }
        const float e = j <= i ? expf(G[i] - G[j]) : 0.f;  // (above the diagonal the exponent may be large)
        L[i * LA + j] = j < i ? beta[i] * e * kk[a][b] : 0.f;
        pt[j * C + i] = e * qk[a][b];
      }
  }
  // e^(G_C - G) K, and e^G Q as columns
  const float last = G[C - 1];
  float* kd = p.kd + at * C * DP;
  for (int i = warp; i < C; i += kPrepareThreads / 32) {
    const float e = expf(last - G[i]);
    for (int d = lane; d < DP; d += 32) kd[i * DP + d] = ks[i * LD + d] * e;
  }
  float* wq = p.wq + at * DP * 2 * C;
  for (int i = warp * 4; i < C; i += kPrepareThreads / 8)
    for (int d = lane; d < DP; d += 32)
      *reinterpret_cast<float4*>(wq + (size_t)d * 2 * C + C + i) =
          make_float4(qs[i * LD + d] * eg[i], qs[(i + 1) * LD + d] * eg[i + 1], qs[(i + 2) * LD + d] * eg[i + 2], qs[(i + 3) * LD + d] * eg[i + 3]);
  if (tid == 0) p.through[at] = eg[C - 1];
  __syncthreads();
  // (I + L) X = diag(beta) [V | e^G K], a column a thread, forward substitution in registers
  for (int c = tid; c < in.V + DP; c += kPrepareThreads) {
    float X[C];
    if (c < in.V) {
      const T* v = (const T*)in.x + (size_t)row0 * in.stride + in.v_off + h * in.V + c;
#pragma unroll
      for (int i = 0; i < C; ++i) X[i] = i < n ? asb::to_float(v[(size_t)i * in.stride]) : 0.f;
#pragma unroll
      for (int i = 0; i < C; ++i) X[i] *= beta[i];
    } else {
#pragma unroll
      for (int i = 0; i < C; ++i) X[i] = beta[i] * eg[i] * ks[i * LD + c - in.V];
    }
#pragma unroll
    for (int i = 1; i < C; ++i) {
      float acc[4] = {X[i], 0.f, 0.f, 0.f};
#pragma unroll
      for (int j = 0; j < i; j += 4) {
        const float4 l = *reinterpret_cast<const float4*>(L + i * LA + j);  // (zeros from the diagonal on)
        acc[0] = fmaf(-l.x, X[j], acc[0]);
        if (j + 1 < i) acc[1] = fmaf(-l.y, X[j + 1], acc[1]);
        if (j + 2 < i) acc[2] = fmaf(-l.z, X[j + 2], acc[2]);
        if (j + 3 < i) acc[3] = fmaf(-l.w, X[j + 3], acc[3]);
      }
      X[i] = (acc[0] + acc[1]) + (acc[2] + acc[3]);
    }
    if (c < in.V) {
      float* y = p.y + at * C * p.VP + c;
#pragma unroll
      for (int i = 0; i < C; ++i) y[(size_t)i * p.VP] = X[i];
    } else {
      float* w = wq + (size_t)(c - in.V) * 2 * C;
#pragma unroll
      for (int i = 0; i < C; i += 4) *reinterpret_cast<float4*>(w + i) = make_float4(X[i], X[i + 1], X[i + 2], X[i + 3]);
    }
  }
}

// acc += A B over k_end (a multiple of 4) values of k, A's rows and B's columns four at a time from shared
// memory, the next four k's operands on their way while these are multiplied
__device__ __forceinline__ void multiply_add(float (&acc)[4][4], const float* a, int a_stride, const float* b, int b_stride, int k_end) {
  float4 av[4], bv[4];
#pragma unroll
  for (int u = 0; u < 4; ++u) {
    av[u] = *reinterpret_cast<const float4*>(a + u * a_stride);
    bv[u] = *reinterpret_cast<const float4*>(b + u * b_stride);
  }
#pragma unroll 2
  for (int k = 0; k < k_end; k += 4) {
    float4 an[4], bn[4];
    const int next = k + 4 < k_end ? k + 4 : 0;  // (past the end: any operands, never used)
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      an[u] = *reinterpret_cast<const float4*>(a + (next + u) * a_stride);
      bn[u] = *reinterpret_cast<const float4*>(b + (next + u) * b_stride);
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float x[4] = {av[u].x, av[u].y, av[u].z, av[u].w}, w[4] = {bv[u].x, bv[u].y, bv[u].z, bv[u].w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], w[j], acc[i][j]);
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      av[u] = an[u];
      bv[u] = bn[u];
    }
  }
}

// count floats (a multiple of 4) into shared memory, asynchronously
template <int THREADS>
__device__ __forceinline__ void fetch(float* dst, const float* src, int count) {
  for (int i = threadIdx.x * 4; i < count; i += THREADS * 4) cp_async16(smem_u32(dst + i), src + i, true);
}

// Two groups of threads, each with a thread per 4 x 4 tile of [W ; Q] S.
template <int C, int VS>
struct Walk {
  static constexpr int kGroup = (2 * C / 4) * (VS / 4), kThreads = 2 * kGroup;
  static constexpr size_t floats(int DP) { return (size_t)DP * 2 * C + (size_t)C * DP + C * C + 4 * C * VS + (size_t)DP * VS; }
};

template <int C, int VS>
__global__ void __launch_bounds__(Walk<C, VS>::kThreads)
delta_chunk_walk_kernel(const ChunkParams p) {
  constexpr int NG = Walk<C, VS>::kGroup, NT = Walk<C, VS>::kThreads, CT = VS / 4;
  extern __shared__ __align__(16) float smem[];
  const DeltaInputs& in = p.in;
  const int DP = p.DP, V = in.V, H = in.H;
  float* wq = smem;                 // [DP][2 C]
  float* kd = wq + DP * 2 * C;      // [C][DP]
  float* pt = kd + C * DP;          // [C][C]
  float* y = pt + C * C;            // [C][VS]
  float* u = y + C * VS;            // [C][VS]
  float* S = u + C * VS;            // [DP][VS]
  float* second = S + DP * VS;      // [2 C][VS]: the second group's share of [W ; Q] S
  asb::pdl_wait();
  asb::pdl_launch_dependents();
  const int tid = threadIdx.x, h = blockIdx.y, v0 = blockIdx.z * VS;
  const int r = p.req[3 * blockIdx.x], c_first = p.req[3 * blockIdx.x + 1], c_end = c_first + p.req[3 * blockIdx.x + 2];
  auto fetch_first = [&](int c) {  // what the products with S read
    const size_t at = (size_t)c * H + h;
    fetch<NT>(wq, p.wq + at * DP * 2 * C, DP * 2 * C);
    const float* ys = p.y + at * C * p.VP + v0;
    for (int i = tid; i < C * CT; i += NT) cp_async16(smem_u32(y + i * 4), ys + (size_t)(i / CT) * p.VP + i % CT * 4, true);
  };
  auto fetch_second = [&](int c) {
    const size_t at = (size_t)c * H + h;
    fetch<NT>(kd, p.kd + at * C * DP, C * DP);
    fetch<NT>(pt, p.pt + at * C * C, C * C);
  };
  fetch_first(c_first);
  cp_async_commit();
  fetch_second(c_first);
  cp_async_commit();
  float* sp = p.state + (((size_t)p.state_slots[r] * H + h) * in.D) * V + v0;
  for (int i = tid; i < DP * VS; i += NT) {
    const int d = i / VS, c = i - d * VS;
    S[i] = (d < in.D && v0 + c < V) ? sp[(size_t)d * V + c] : 0.f;
  }
  // [W ; Q] S: both groups, each over its half of the rows of S; then the first group makes U (its tiles of W)
  // and O (those of Q) and the second the new S
  const bool first = tid < NG;
  const int t = first ? tid : tid - NG, rt = t / CT, ct = t % CT;
  const int k_half = (DP / 4 + 1) / 2 * 4, k_from = first ? 0 : k_half, k_count = first ? k_half : DP - k_half;
  for (int c = c_first; c < c_end; ++c) {
    const int row0 = p.chunk_row[c], n = p.chunk_len[c];
    const float through = p.through[(size_t)c * H + h];
    cp_async_wait<1>();
    __syncthreads();
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    if (k_count > 0) multiply_add(acc, wq + k_from * 2 * C + rt * 4, 2 * C, S + k_from * VS + ct * 4, VS, k_count);
    if (!first) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        *reinterpret_cast<float4*>(second + (rt * 4 + i) * VS + ct * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    }
    __syncthreads();  // W and Q have been read
    if (first) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int at = (rt * 4 + i) * VS + ct * 4;
        const float4 rest = *reinterpret_cast<const float4*>(second + at);
        acc[i][0] += rest.x; acc[i][1] += rest.y; acc[i][2] += rest.z; acc[i][3] += rest.w;
        if (rt < C / 4) {
          const float4 own = *reinterpret_cast<const float4*>(y + at);
          *reinterpret_cast<float4*>(u + at) = make_float4(own.x - acc[i][0], own.y - acc[i][1], own.z - acc[i][2], own.w - acc[i][3]);
        }
      }
    }
    cp_async_wait<0>();  // (K and P of this chunk)
    __syncthreads();     // U is there, and Y has been read
    if (c + 1 < c_end) fetch_first(c + 1);
    cp_async_commit();
    if (!first) {
      for (int tile = t; tile < DP / 4 * CT; tile += NG) {
        const int d0 = tile / CT * 4, c0 = tile % CT * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 s = *reinterpret_cast<const float4*>(S + (d0 + i) * VS + c0);
          acc[i][0] = through * s.x; acc[i][1] = through * s.y; acc[i][2] = through * s.z; acc[i][3] = through * s.w;
        }
        multiply_add(acc, kd + d0, DP, u + c0, VS, C);
#pragma unroll
        for (int i = 0; i < 4; ++i)
          *reinterpret_cast<float4*>(S + (d0 + i) * VS + c0) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
      }
    } else if (rt >= C / 4) {
      const int i0 = rt * 4 - C;
      multiply_add(acc, pt + i0, C, u + ct * 4, VS, C);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (i0 + i >= n) break;
        float* o = p.out + ((size_t)(row0 + i0 + i) * H + h) * V + v0 + ct * 4;
        if (V % 4 == 0) {
          if (v0 + ct * 4 < V) *reinterpret_cast<float4*>(o) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (v0 + ct * 4 + j < V) o[j] = acc[i][j];
        }
      }
    }
    __syncthreads();  // S is new, and K, P and U have been read
    if (c + 1 < c_end) fetch_second(c + 1);
    cp_async_commit();
  }
  cp_async_wait<0>();
  for (int i = tid; i < DP * VS; i += NT) {
    const int d = i / VS, c = i - d * VS;
    if (d < in.D && v0 + c < V) sp[(size_t)d * V + c] = S[i];
  }
}

template <int C, int VS>
int launch_walk(const ChunkParams& p, int n, cudaStream_t stream) {
  const size_t smem = sizeof(float) * Walk<C, VS>::floats(p.DP);
  auto kern = delta_chunk_walk_kernel<C, VS>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return asb::fail("delta_chunks: shared memory %zu: %s", smem, cudaGetErrorString(e));
  dim3 grid(n, p.in.H, (p.in.V + VS - 1) / VS);
  asb::launch(kern, grid, Walk<C, VS>::kThreads, smem, stream, p);
  return asb::check_launch("delta_chunk_walk");
}

template <typename T, int C>
int launch_chunks(const ChunkParams& p, int chunks, int n, cudaStream_t stream) {
  const size_t smem = sizeof(float) * (2 * (size_t)C * (p.DP + 4) + C * (C + 4) + 3 * C);
  auto kern = delta_chunk_prepare_kernel<T, C>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return asb::fail("delta_chunks: shared memory %zu: %s", smem, cudaGetErrorString(e));
  asb::launch(kern, dim3(chunks, p.in.H), kPrepareThreads, smem, stream, p);
  if (int rc = asb::check_launch("delta_chunk_prepare")) return rc;
  // narrower slices of the value columns where wide ones would leave SMs without a block
  if ((long long)n * p.in.H * ((p.in.V + 31) / 32) < 148) return launch_walk<C, 16>(p, n, stream);
  return launch_walk<C, 32>(p, n, stream);
}

int check_inputs(const DeltaInputs& in, const char* what) {
  if (in.H < 1 || in.D < 1 || in.V < 1 || in.H > 65535) return asb::fail("%s: %d heads of %d x %d", what, in.H, in.D, in.V);
  if (in.share < 1 || in.H % in.share) return asb::fail("%s: %d heads do not share q and k in groups of %d", what, in.H, in.share);
  return 0;
}

DeltaInputs inputs(const void* x, int stride, int q_off, int k_off, int v_off, const float* z, int z_stride, int b_off, int a_off,
                   const float* dt_bias, const float* a_log, int H, int D, int V, int share, float q_scale) {
  DeltaInputs in;
  in.x = x; in.z = z; in.dt_bias = dt_bias; in.a_log = a_log; in.stride = stride; in.q_off = q_off; in.k_off = k_off; in.v_off = v_off;
  in.z_stride = z_stride; in.b_off = b_off; in.a_off = a_off; in.H = H; in.D = D; in.V = V; in.share = share; in.q_scale = q_scale;
  return in;
}

}  // namespace

// Tokens a chunk holds for keys of D entries (0: keys too long for asb_delta_chunks; every portion then
// runs token by token).
extern "C" int asb_delta_chunk_tokens(int D) { return D <= 128 ? 64 : (D <= 256 ? 32 : 0); }

// limit > 0: requests that bring more than `limit` tokens are skipped.
extern "C" int asb_delta_step(float* out, const void* x, int stride, int q_off, int k_off, int v_off, const float* z, int z_stride,
                              int b_off, int a_off, const float* dt_bias, const float* a_log, float* state, const int* state_slots,
                              const int* req_q_start, int R, int H, int D, int V, int share, float q_scale, int limit, int dtype,
                              cudaStream_t stream) {
  if (R == 0) return 0;
  StepParams p;
  p.in = inputs(x, stride, q_off, k_off, v_off, z, z_stride, b_off, a_off, dt_bias, a_log, H, D, V, share, q_scale);
  if (int rc = check_inputs(p.in, "delta_step")) return rc;
  if (D > 1024) return asb::fail("delta_step: key size %d exceeds 1024", D);
  p.out = out; p.state = state; p.state_slots = state_slots; p.req_q_start = req_q_start; p.limit = limit;
  int cv = V > 64 ? 4 : (V > 32 ? 2 : 1);
  while (cv > 1 && (V % cv || ((uintptr_t)state | (uintptr_t)out) % (4 * cv))) cv >>= 1;
  if ((V + 32 * cv - 1) / (32 * cv) > 65535) return asb::fail("delta_step: value size %d", V);
  ASB_DISPATCH_DTYPE(dtype, T, {
    if (D <= 32) return launch_step_columns<T, 4>(p, R, cv, stream);
    if (D <= 128) return launch_step_columns<T, 16>(p, R, cv, stream);
    if (D <= 256) return launch_step_columns<T, 32>(p, R, cv, stream);
    return launch_step<T, 128, 1>(p, R, stream);
  });
  return 0;
}

// chunk_row, chunk_len [chunks]; req [n, 3] (request, first chunk, chunks), the requests' chunks in order.
// The workspaces hold chunks * H blocks each: wq DP * 2 C, kd C * DP, pt C * C, y C * VP and through 1
// floats, with C = asb_delta_chunk_tokens(D), DP = D to a multiple of 4, VP = V to a multiple of 32.
extern "C" int asb_delta_chunks(float* out, const void* x, int stride, int q_off, int k_off, int v_off, const float* z, int z_stride,
                                int b_off, int a_off, const float* dt_bias, const float* a_log, float* state, const int* state_slots,
                                const int* chunk_row, const int* chunk_len, const int* req, float* wq, float* kd, float* pt, float* y,
                                float* through, int chunks, int n, int H, int D, int V, int share, float q_scale, int dtype,
                                cudaStream_t stream) {
  if (chunks == 0 || n == 0) return 0;
  ChunkParams p;
  p.in = inputs(x, stride, q_off, k_off, v_off, z, z_stride, b_off, a_off, dt_bias, a_log, H, D, V, share, q_scale);
  if (int rc = check_inputs(p.in, "delta_chunks")) return rc;
  const int C = asb_delta_chunk_tokens(D);
  if (C == 0) return asb::fail("delta_chunks: key size %d exceeds 256", D);
  if (((uintptr_t)out | (uintptr_t)wq | (uintptr_t)kd | (uintptr_t)pt | (uintptr_t)y) & 15) return asb::fail("delta_chunks: unaligned buffers");
  if ((V + 15) / 16 > 65535) return asb::fail("delta_chunks: value size %d", V);
  p.out = out; p.state = state; p.state_slots = state_slots; p.chunk_row = chunk_row; p.chunk_len = chunk_len; p.req = req;
  p.wq = wq; p.kd = kd; p.pt = pt; p.y = y; p.through = through;
  p.DP = (D + 3) / 4 * 4; p.VP = (V + 31) / 32 * 32;
  ASB_DISPATCH_DTYPE(dtype, T, {
    if (C == 64) return launch_chunks<T, 64>(p, chunks, n, stream);
    return launch_chunks<T, 32>(p, chunks, n, stream);
  });
  return 0;
}
