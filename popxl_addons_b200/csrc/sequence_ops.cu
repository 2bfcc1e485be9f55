// Kernels of sequence models that keep a 32-bit residual stream and per-sequence state:
//   xl_embed_dyt        x = table[token] (fp32) and h = DyT(x), the first normalised activations
//   xl_residual_dyt     x += mult * y (+ table[token]) and h = DyT(x) of the updated stream, one pass
//   xl_select_dyt       DyT of selected rows of the stream (the rows whose logits are asked for)
//   xl_swiglu_packed    silu(gate) * up on rows [gate | up]
//   xl_min_gru          gated linear recurrence S_t = (1 - z_t) S_{t-1} + z_t c_t over a portion of every sequence
//   xl_advance_by       pos[b] += count[b]
// Dynamic Tanh (DyT): tanh(alpha * x) * w + b, element by element, so it folds into whatever produced x.
// Rows of a portion are (sequence, token) with `T` tokens per sequence; `count[b]` of them are real, the rest is padding.
#include "common.cuh"

#include <cooperative_groups.h>
#include <math.h>

namespace cg = cooperative_groups;

namespace {

// V consecutive elements, V * sizeof(T) bytes, naturally aligned
template <typename T, int V> struct alignas(V * sizeof(T)) Pack { T v[V]; };
template <typename T, int V> __device__ __forceinline__ void load_pack(const T* p, float (&o)[V]) {
  const Pack<T, V> r = *reinterpret_cast<const Pack<T, V>*>(p);
#pragma unroll
  for (int i = 0; i < V; ++i) o[i] = xl_to_float(r.v[i]);
}
template <typename T, int V> __device__ __forceinline__ void store_pack(T* p, const float (&o)[V]) {
  Pack<T, V> r;
#pragma unroll
  for (int i = 0; i < V; ++i) r.v[i] = xl_from_float<T>(o[i]);
  *reinterpret_cast<Pack<T, V>*>(p) = r;
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }

struct DytParams {
  const float* alpha;  // one value; null: no norm follows
  const float* w;
  const float* b;
};

template <int V>
__device__ __forceinline__ void dyt_pack(const float (&x)[V], float alpha, const DytParams& n, int c, float (&h)[V]) {
  float w[V], b[V];
  load_pack<float, V>(n.w + c, w);
  load_pack<float, V>(n.b + c, b);
#pragma unroll
  for (int i = 0; i < V; ++i) h[i] = tanhf(alpha * x[i]) * w[i] + b[i];
}

// x (rows, cols) fp32 += mult * y, then += table[token] where a table is given; h = DyT(x). Without y, x is overwritten by
// the table row (embedding).
template <typename T, int V>
__global__ void __launch_bounds__(256)
    stream_dyt_kernel(float* __restrict__ x, const T* __restrict__ y, float mult, const int* __restrict__ tokens,
                      const T* __restrict__ table, int vocab, DytParams n, T* __restrict__ h, long long rows, int cols) {
  const float alpha = n.alpha ? *n.alpha : 0.f;
  const int per_row = cols / V;
  const long long total = rows * per_row;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long row = i / per_row;
    const int c = (int)(i - row * per_row) * V;
    const long long off = row * cols + c;
    float v[V];
    if (y) {
      float d[V];
      load_pack<float, V>(x + off, v);
      load_pack<T, V>(y + off, d);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += mult * d[e];
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = 0.f;
    }
    if (table) {
      const int t = min(max(tokens[row], 0), vocab - 1);
      float d[V];
      load_pack<T, V>(table + (long long)t * cols + c, d);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] += d[e];
    }
    store_pack<float, V>(x + off, v);
    if (n.alpha) {
      float o[V];
      dyt_pack<V>(v, alpha, n, c, o);
      store_pack<T, V>(h + off, o);
    }
  }
}

// h[r] = DyT(x[r * stride + idx[r] - offset])
template <typename T>
__global__ void __launch_bounds__(256)
    select_dyt_kernel(const float* __restrict__ x, const int* __restrict__ idx, int stride, int offset, long long x_rows,
                      DytParams n, T* __restrict__ h, int cols) {
  const float alpha = *n.alpha;
  const long long r = blockIdx.x;
  long long src = r * stride + idx[r] - offset;
  src = src < 0 ? 0 : (src >= x_rows ? x_rows - 1 : src);
  for (int c = threadIdx.x; c < cols; c += blockDim.x)
    h[r * cols + c] = xl_from_float<T>(tanhf(alpha * x[src * cols + c]) * n.w[c] + n.b[c]);
}

template <typename T, int V>
__global__ void __launch_bounds__(256) swiglu_packed_kernel(const T* __restrict__ gu, T* __restrict__ y, long long rows, int F) {
  const int per_row = F / V;
  const long long total = rows * per_row;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long row = i / per_row;
    const int c = (int)(i - row * per_row) * V;
    float g[V], u[V];
    load_pack<T, V>(gu + row * 2 * F + c, g);
    load_pack<T, V>(gu + row * 2 * F + F + c, u);
#pragma unroll
    for (int e = 0; e < V; ++e) g[e] = silu_f(g[e]) * u[e];
    store_pack<T, V>(y + row * F + c, g);
  }
}

__global__ void advance_by_kernel(int* pos, const int* count, int n) {
  for (int i = threadIdx.x; i < n; i += blockDim.x) pos[i] += count[i];
}

// ------------------------------------------------------------------------------------------------------------------
// minGRU over a portion. zxg: (B*T, 3W) rows [z | candidate | output gate] pre-activations without biases. Every channel
// is an independent first-order recurrence, and composing steps is associative: (a, b) then (a', b') = (a a', a' b + b').
// A CTA owns 32*V channels and 16 warps x 8 tokens; a cluster of CTAs covers consecutive token ranges of the same channels
// and exchanges the range totals through distributed shared memory, so all operands are read from memory exactly once.
// The state (B, W) stays in fp32; a sequence at position 0 starts from zero whatever the state buffer holds.
// ------------------------------------------------------------------------------------------------------------------
constexpr int GRU_WARPS = 16;
constexpr int GRU_STEPS = 8;
constexpr int GRU_TILE = GRU_WARPS * GRU_STEPS;  // tokens per CTA and iteration
constexpr int GRU_MAX_CLUSTER = 8;

template <typename T, int V>
__global__ void __launch_bounds__(GRU_WARPS * 32)
    min_gru_kernel(const T* __restrict__ zxg, const float* __restrict__ bz, const float* __restrict__ bx,
                   float* __restrict__ state, T* __restrict__ y, const int* __restrict__ pos, const int* __restrict__ count,
                   int T_len, int W) {
  __shared__ float2 part[GRU_WARPS][32 * V];
  __shared__ float2 total[2][32 * V];  // double-buffered: a CTA of the cluster may still read the previous iteration's
  cg::cluster_group cluster = cg::this_cluster();
  const int C = (int)cluster.num_blocks(), rank = (int)cluster.block_rank();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int b = blockIdx.z;
  const int ch = (blockIdx.y * 32 + lane) * V;
  const bool on = ch < W;  // W is a multiple of V
  const int cnt = min(count[b], T_len);
  float bzv[V], bxv[V], carry[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    bzv[e] = on ? bz[ch + e] : 0.f;
    bxv[e] = on ? bx[ch + e] : 0.f;
    carry[e] = (on && pos[b] > 0) ? state[(long long)b * W + ch + e] : 0.f;
  }
  int buf = 0;
  for (int t0 = 0; t0 < cnt; t0 += C * GRU_TILE, buf ^= 1) {
    const int t_first = t0 + rank * GRU_TILE + warp * GRU_STEPS;
    float a[GRU_STEPS][V], bb[GRU_STEPS][V], g[GRU_STEPS][V];
#pragma unroll
    for (int s = 0; s < GRU_STEPS; ++s) {
      if (on && t_first + s < cnt) {
        const T* row = zxg + ((long long)b * T_len + t_first + s) * 3 * W + ch;
        load_pack<T, V>(row, a[s]);
        load_pack<T, V>(row + W, bb[s]);
        load_pack<T, V>(row + 2 * W, g[s]);
      } else {
#pragma unroll
        for (int e = 0; e < V; ++e) a[s][e] = bb[s][e] = g[s][e] = 0.f;
      }
    }
    float A[V], B[V];
#pragma unroll
    for (int e = 0; e < V; ++e) { A[e] = 1.f; B[e] = 0.f; }
#pragma unroll
    for (int s = 0; s < GRU_STEPS; ++s) {
      const bool real = t_first + s < cnt;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float z = sigmoid_f(a[s][e] + bzv[e]);
        const float u = bb[s][e] + bxv[e];
        const float c = u >= 0.f ? u + 0.5f : sigmoid_f(u);
        a[s][e] = real ? 1.f - z : 1.f;
        bb[s][e] = real ? z * c : 0.f;
        B[e] = a[s][e] * B[e] + bb[s][e];
        A[e] *= a[s][e];
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) part[warp][lane * V + e] = make_float2(A[e], B[e]);
    __syncthreads();
    if (warp == GRU_WARPS - 1) {
#pragma unroll
      for (int e = 0; e < V; ++e) {
        float2 acc = make_float2(1.f, 0.f);
        for (int w = 0; w < GRU_WARPS; ++w) {
          const float2 p = part[w][lane * V + e];
          acc = make_float2(acc.x * p.x, p.x * acc.y + p.y);
        }
        total[buf][lane * V + e] = acc;
      }
    }
    cluster.sync();
    float S[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      S[e] = carry[e];
      for (int r = 0; r < C; ++r) {
        const float2 p = cluster.map_shared_rank(&total[buf][0], r)[lane * V + e];
        if (r == rank) S[e] = carry[e];
        carry[e] = p.x * carry[e] + p.y;
      }
      for (int w = 0; w < warp; ++w) {
        const float2 p = part[w][lane * V + e];
        S[e] = p.x * S[e] + p.y;
      }
    }
#pragma unroll
    for (int s = 0; s < GRU_STEPS; ++s) {
      float o[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        S[e] = a[s][e] * S[e] + bb[s][e];
        o[e] = S[e] * silu_f(g[s][e]);
      }
      if (on && t_first + s < cnt) store_pack<T, V>(y + ((long long)b * T_len + t_first + s) * W + ch, o);
    }
    __syncthreads();  // `part` is rewritten by the next iteration
  }
  if (rank == 0 && warp == 0 && on) {
#pragma unroll
    for (int e = 0; e < V; ++e) state[(long long)b * W + ch + e] = carry[e];
  }
  cluster.sync();  // no CTA leaves while another may still read its totals
}

template <typename T, int V>
int launch_min_gru(const void* zxg, const float* bz, const float* bx, float* state, void* y, const int* pos, const int* count,
                   int B, int T_len, int W, cudaStream_t s) {
  const int groups = (W + 32 * V - 1) / (32 * V);
  int C = 1;
  while (C < GRU_MAX_CLUSTER && C * GRU_TILE < T_len && (long long)groups * B * C < 2 * 148) C *= 2;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(C, groups, B);
  cfg.blockDim = dim3(GRU_WARPS * 32);
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = C;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  const cudaError_t e = cudaLaunchKernelEx(&cfg, min_gru_kernel<T, V>, (const T*)zxg, bz, bx, state, (T*)y, pos, count, T_len, W);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

template <typename T>
int launch_stream(float* x, const void* y, float mult, const int* tokens, const void* table, int vocab, DytParams n, void* h,
                  long long rows, int cols, cudaStream_t s) {
  if (cols % 4 == 0) {
    stream_dyt_kernel<T, 4><<<xl_grid_for(rows * (cols / 4), 256), 256, 0, s>>>(x, (const T*)y, mult, tokens, (const T*)table,
                                                                               vocab, n, (T*)h, rows, cols);
  } else {
    stream_dyt_kernel<T, 1><<<xl_grid_for(rows * cols, 256), 256, 0, s>>>(x, (const T*)y, mult, tokens, (const T*)table, vocab,
                                                                         n, (T*)h, rows, cols);
  }
  return (int)cudaGetLastError();
}

}  // namespace

// x (rows, cols) fp32; y, h, table of type `dtype`. y null: x = table[tokens] (embedding). table null: no row is added.
// alpha null: no norm (h unused), else h = tanh(alpha x) w + b. All base pointers 16-byte aligned.
XL_API int xl_stream_dyt(float* x, const void* y, float mult, const int* tokens, const void* table, int vocab,
                         const float* alpha, const float* w, const float* b, void* h, long long rows, int cols, int dtype,
                         cudaStream_t s) {
  if (rows < 1 || cols < 1 || (!y && !table) || (table && (!tokens || vocab < 1)) || (alpha && (!w || !b || !h))) return -1;
  const DytParams n{alpha, w, b};
  XL_DISPATCH_DTYPE(dtype, T, { return launch_stream<T>(x, y, mult, tokens, table, vocab, n, h, rows, cols, s); });
  return (int)cudaGetLastError();
}

XL_API int xl_select_dyt(const float* x, const int* idx, int stride, int offset, long long x_rows, const float* alpha,
                         const float* w, const float* b, void* h, int rows, int cols, int dtype, cudaStream_t s) {
  if (rows < 1 || cols < 1 || x_rows < 1 || !alpha || !w || !b) return -1;
  const DytParams n{alpha, w, b};
  XL_DISPATCH_DTYPE(dtype, T, {
    select_dyt_kernel<T><<<rows, 256, 0, s>>>(x, idx, stride, offset, x_rows, n, (T*)h, cols);
  });
  return (int)cudaGetLastError();
}

// gu: (rows, 2F) rows [gate | up]; y: (rows, F)
XL_API int xl_swiglu_packed(const void* gu, void* y, long long rows, int F, int dtype, cudaStream_t s) {
  if (rows < 1 || F < 1) return -1;
  XL_DISPATCH_DTYPE(dtype, T, {
    constexpr int V = 16 / sizeof(T);
    if (F % V == 0)
      swiglu_packed_kernel<T, V><<<xl_grid_for(rows * (F / V), 256), 256, 0, s>>>((const T*)gu, (T*)y, rows, F);
    else
      swiglu_packed_kernel<T, 1><<<xl_grid_for(rows * F, 256), 256, 0, s>>>((const T*)gu, (T*)y, rows, F);
  });
  return (int)cudaGetLastError();
}

XL_API int xl_advance_by(int* pos, const int* count, int n, cudaStream_t s) {
  advance_by_kernel<<<1, 128, 0, s>>>(pos, count, n);
  return (int)cudaGetLastError();
}

// zxg (B*T_len, 3W) and y (B*T_len, W) of type `dtype`; bz, bx (W), state (B, W) fp32; pos, count (B) int32.
XL_API int xl_min_gru(const void* zxg, const float* bz, const float* bx, float* state, void* y, const int* pos, const int* count,
                      int B, int T_len, int W, int dtype, cudaStream_t s) {
  if (B < 1 || B > 65535 || T_len < 1 || W < 1 || (W + 31) / 32 > 65535) return -1;
  XL_DISPATCH_DTYPE(dtype, T, {
    return W % 2 == 0 ? launch_min_gru<T, 2>(zxg, bz, bx, state, y, pos, count, B, T_len, W, s)
                      : launch_min_gru<T, 1>(zxg, bz, bx, state, y, pos, count, B, T_len, W, s);
  });
  return (int)cudaGetLastError();
}
