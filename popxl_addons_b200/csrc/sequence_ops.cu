// Kernels of sequence models that keep a 32-bit residual stream and per-sequence state:
//   xl_embed_dyt        x = table[token] (fp32) and h = DyT(x), the first normalised activations
//   xl_residual_dyt     x += mult * y (+ table[token]) and h = DyT(x) of the updated stream, one pass
//   xl_select_dyt       DyT of selected rows of the stream (the rows whose logits are asked for)
//   xl_stream_rms       x = scale * table[token], or x += mult * y, and h = the RMS norm of the updated stream, one pass
//   xl_select_rms       RMS norm of selected rows of the stream
//   xl_swiglu_packed    silu(gate) * up on rows [gate | up]
//   xl_clamped_glu      g * sigmoid(slope g) * (u + shift) of clamped gate and up columns of wider rows
//   xl_min_gru          gated linear recurrence S_t = (1 - z_t) S_{t-1} + z_t c_t over a portion of every sequence
//   xl_advance_by       pos[b] += count[b]
// Dynamic Tanh (DyT): tanh(alpha * x) * w + b, element by element, so it folds into whatever produced x.
// Rows of a portion are (sequence, token) with `T` tokens per sequence; `count[b]` of them are real, the rest is padding.
#include "common.cuh"

#include <math.h>

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

// ---- RMS norm: one CTA per row, the row in registers between the sum of squares and the output --------------------------
constexpr int RMS_THREADS = 256;

// x (rows, cols) fp32 += mult * y, or without y: x = mult * table[token]; with w, h = x / sqrt(mean(x^2) + eps) * w.
// NP packs of V columns per thread stay in registers; the columns of longer rows are read again.
template <typename T, int V, int NP>
__global__ void __launch_bounds__(RMS_THREADS)
    stream_rms_kernel(float* __restrict__ x, const T* __restrict__ y, float mult, const int* __restrict__ tokens,
                      const T* __restrict__ table, int vocab, const float* __restrict__ w, float eps, T* __restrict__ h, int cols) {
  __shared__ float red[32];
  const long long row = blockIdx.x;
  float* xr = x + row * cols;
  const T* src = y ? y + row * cols : table + (long long)min(max(tokens[row], 0), vocab - 1) * cols;
  const int step = blockDim.x * V, c0 = threadIdx.x * V;
  float keep[NP][V], sq = 0.f;
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int c = c0 + i * step;
    if (c < cols) {
      float d[V];
      load_pack<T, V>(src + c, d);
      if (y) load_pack<float, V>(xr + c, keep[i]);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        keep[i][e] = y ? keep[i][e] + mult * d[e] : mult * d[e];
        sq += keep[i][e] * keep[i][e];
      }
      store_pack<float, V>(xr + c, keep[i]);
    }
  }
  for (int c = c0 + NP * step; c < cols; c += step) {
    float d[V], v[V];
    load_pack<T, V>(src + c, d);
    if (y) load_pack<float, V>(xr + c, v);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      v[e] = y ? v[e] + mult * d[e] : mult * d[e];
      sq += v[e] * v[e];
    }
    store_pack<float, V>(xr + c, v);
  }
  if (!w) return;
  const float f = 1.f / sqrtf(xl_block_sum(sq, red) / cols + eps);
  T* hr = h + row * cols;
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int c = c0 + i * step;
    if (c < cols) {
      float g[V];
      load_pack<float, V>(w + c, g);
#pragma unroll
      for (int e = 0; e < V; ++e) g[e] *= keep[i][e] * f;
      store_pack<T, V>(hr + c, g);
    }
  }
  for (int c = c0 + NP * step; c < cols; c += step) {
    float g[V], v[V];
    load_pack<float, V>(w + c, g);
    load_pack<float, V>(xr + c, v);  // written by this thread
#pragma unroll
    for (int e = 0; e < V; ++e) g[e] *= v[e] * f;
    store_pack<T, V>(hr + c, g);
  }
}

// h[r] = RMS norm of x[r * stride + idx[r] - offset]
template <typename T>
__global__ void __launch_bounds__(RMS_THREADS)
    select_rms_kernel(const float* __restrict__ x, const int* __restrict__ idx, int stride, int offset, long long x_rows,
                      const float* __restrict__ w, float eps, T* __restrict__ h, int cols) {
  __shared__ float red[32];
  const long long r = blockIdx.x;
  long long src = r * stride + idx[r] - offset;
  src = src < 0 ? 0 : (src >= x_rows ? x_rows - 1 : src);
  const float* xr = x + src * cols;
  float sq = 0.f;
  for (int c = threadIdx.x; c < cols; c += blockDim.x) sq += xr[c] * xr[c];
  const float f = 1.f / sqrtf(xl_block_sum(sq, red) / cols + eps);
  for (int c = threadIdx.x; c < cols; c += blockDim.x) h[r * cols + c] = xl_from_float<T>(xr[c] * f * w[c]);
}

// gate: columns [0, F) of rows of stride ldg, up: the F columns after them; y: F columns of rows of stride ldy.
template <typename T, int V>
__global__ void __launch_bounds__(256)
    clamped_glu_kernel(const T* __restrict__ gate, long long ldg, T* __restrict__ y, long long ldy, long long rows, int F,
                       float limit, float slope, float shift) {
  const int per_row = F / V;
  const long long total = rows * per_row;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long row = i / per_row;
    const int c = (int)(i - row * per_row) * V;
    float g[V], u[V];
    load_pack<T, V>(gate + row * ldg + c, g);
    load_pack<T, V>(gate + row * ldg + F + c, u);
#pragma unroll
    for (int e = 0; e < V; ++e) g[e] = xl_clamped_glu_value(g[e], u[e], limit, slope, shift);
    store_pack<T, V>(y + row * ldy + c, g);
  }
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
// The portion is cut into ranges of `L` tokens. The first kernel composes every range but the last to one (a, b) per channel;
// in the second, each range folds its predecessors' pairs onto the state it starts from and walks its tokens. A portion of
// one range needs only the second. One thread per range and V channels; loads of GRU_AHEAD tokens are in flight together.
// The state (B, W) stays in fp32; a sequence at position 0 starts from zero whatever the state buffer holds. All ranges read
// the old state, so the new one waits in the last slot of `pairs` until a third, tiny kernel stores it.
// ------------------------------------------------------------------------------------------------------------------
constexpr int GRU_THREADS = 128;
constexpr int GRU_AHEAD = 8;
constexpr int GRU_MAX_RANGES = 64;

// 32-bit models: the correctly rounded forms; 16-bit models: the same functions by the hardware's exponential and division
template <typename T> __device__ __forceinline__ float gate_sigmoid(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
template <> __device__ __forceinline__ float gate_sigmoid<float>(float x) { return sigmoid_f(x); }

struct GruParams {
  const float *bz, *bx;
  float* state;
  float2* pairs;  // [B][ranges][W]
  const int *pos, *count;
  int T, W, L, ranges;
};

template <typename T, int V>
__device__ __forceinline__ void gru_step(const float (&zr)[V], const float (&ur)[V], const float (&bz)[V], const float (&bx)[V],
                                         float (&a)[V], float (&b)[V]) {
#pragma unroll
  for (int e = 0; e < V; ++e) {
    const float z = gate_sigmoid<T>(zr[e] + bz[e]), u = ur[e] + bx[e];
    a[e] = 1.f - z;
    b[e] = z * (u >= 0.f ? u + 0.5f : gate_sigmoid<T>(u));
  }
}

template <typename T, int V, bool OUTPUT>
__global__ void __launch_bounds__(GRU_THREADS) min_gru_kernel(const T* __restrict__ zxg, T* __restrict__ y, const GruParams p) {
  const int ch = (blockIdx.x * GRU_THREADS + threadIdx.x) * V;
  const int range = blockIdx.y, b = blockIdx.z;
  const int cnt = min(p.count[b], p.T);
  const int t0 = range * p.L, t1 = min(cnt, t0 + p.L);
  if (ch >= p.W || t0 >= t1) return;
  const long long W = p.W;
  float bz[V], bx[V], S[V], A[V];
  load_pack<float, V>(p.bz + ch, bz);
  load_pack<float, V>(p.bx + ch, bx);
#pragma unroll
  for (int e = 0; e < V; ++e) { S[e] = 0.f; A[e] = 1.f; }
  if (OUTPUT) {
    if (p.pos[b] > 0) load_pack<float, V>(p.state + b * W + ch, S);
    const float2* src = p.pairs + (long long)b * p.ranges * W + ch;
#pragma unroll 4
    for (int r = 0; r < range; ++r) {
      float ab[2 * V];
      load_pack<float, 2 * V>(reinterpret_cast<const float*>(src + r * W), ab);
#pragma unroll
      for (int e = 0; e < V; ++e) S[e] = ab[2 * e] * S[e] + ab[2 * e + 1];
    }
  }
  const T* row = zxg + ((long long)b * p.T + t0) * 3 * W + ch;
  T* out = OUTPUT ? y + ((long long)b * p.T + t0) * W + ch : nullptr;
  for (int t = t0; t < t1; t += GRU_AHEAD) {
    float z[GRU_AHEAD][V], u[GRU_AHEAD][V], g[GRU_AHEAD][V];
#pragma unroll
    for (int i = 0; i < GRU_AHEAD; ++i) {
      const T* src = row + (long long)(t - t0 + (t + i < t1 ? i : 0)) * 3 * W;
      load_pack<T, V>(src, z[i]);
      load_pack<T, V>(src + W, u[i]);
      if (OUTPUT) load_pack<T, V>(src + 2 * W, g[i]);
    }
#pragma unroll
    for (int i = 0; i < GRU_AHEAD; ++i) {
      if (t + i < t1) {
        float a[V], c[V];
        gru_step<T, V>(z[i], u[i], bz, bx, a, c);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          S[e] = a[e] * S[e] + c[e];
          A[e] *= a[e];
        }
        if (OUTPUT) {
          float o[V];
#pragma unroll
          for (int e = 0; e < V; ++e) o[e] = S[e] * g[i][e] * gate_sigmoid<T>(g[i][e]);
          store_pack<T, V>(out + (long long)(t - t0 + i) * W, o);
        }
      }
    }
  }
  if (OUTPUT) {
    // the state at the end of the portion, after the last pair of this sequence (ranges of other CTAs still read `state`)
    if (t1 == cnt) {
      float s2[2 * V];
#pragma unroll
      for (int e = 0; e < V; ++e) { s2[2 * e] = 0.f; s2[2 * e + 1] = S[e]; }
      store_pack<float, 2 * V>(reinterpret_cast<float*>(p.pairs + ((long long)b * p.ranges + p.ranges - 1) * W + ch), s2);
    }
  } else {
    float ab[2 * V];
#pragma unroll
    for (int e = 0; e < V; ++e) { ab[2 * e] = A[e]; ab[2 * e + 1] = S[e]; }
    store_pack<float, 2 * V>(reinterpret_cast<float*>(p.pairs + ((long long)b * p.ranges + range) * W + ch), ab);
  }
}

__global__ void __launch_bounds__(256) min_gru_commit_kernel(const GruParams p) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, b = blockIdx.y;
  if (c < p.W && min(p.count[b], p.T) > 0)
    p.state[(long long)b * p.W + c] = p.pairs[((long long)b * p.ranges + p.ranges - 1) * p.W + c].y;
}

inline int gru_range(int T) {
  int L = (T + GRU_MAX_RANGES - 2) / (GRU_MAX_RANGES - 1);  // one slot of `pairs` is left for the final state
  L = (L + GRU_AHEAD - 1) / GRU_AHEAD * GRU_AHEAD;
  return L < 32 ? 32 : L;
}

template <typename T, int V>
int launch_min_gru(const void* zxg, void* y, GruParams p, int B, cudaStream_t s) {
  const int used = (p.T + p.L - 1) / p.L;
  const dim3 block(GRU_THREADS);
  const int gx = (p.W + V * GRU_THREADS - 1) / (V * GRU_THREADS);
  if (used > 1) min_gru_kernel<T, V, false><<<dim3(gx, used - 1, B), block, 0, s>>>((const T*)zxg, (T*)y, p);
  min_gru_kernel<T, V, true><<<dim3(gx, used, B), block, 0, s>>>((const T*)zxg, (T*)y, p);
  min_gru_commit_kernel<<<dim3((p.W + 255) / 256, B), 256, 0, s>>>(p);
  return (int)cudaGetLastError();
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

template <typename T, int V>
int launch_rms(float* x, const void* y, float mult, const int* tokens, const void* table, int vocab, const float* w, float eps,
               void* h, long long rows, int cols, cudaStream_t s) {
  const int packs = (cols + V - 1) / V;
  const int threads = packs >= RMS_THREADS ? RMS_THREADS : (packs + 31) / 32 * 32;
#define XL_RMS(NP)                                                                                                         \
  stream_rms_kernel<T, V, NP><<<(unsigned)rows, threads, 0, s>>>(x, (const T*)y, mult, tokens, (const T*)table, vocab, w,    \
                                                                 eps, (T*)h, cols)
  if (packs <= RMS_THREADS) XL_RMS(1);
  else if (packs <= 4 * RMS_THREADS) XL_RMS(4);
  else XL_RMS(8);
#undef XL_RMS
  return (int)cudaGetLastError();
}

}  // namespace

// x (rows, cols) fp32; y, h, table of type `dtype`. y null: x = mult * table[tokens] (embedding), else x += mult * y. w null: no
// norm (h unused), else h = x / sqrt(mean(x^2) + eps) * w, w fp32. All base pointers 16-byte aligned.
XL_API int xl_stream_rms(float* x, const void* y, float mult, const int* tokens, const void* table, int vocab, const float* w,
                         float eps, void* h, long long rows, int cols, int dtype, cudaStream_t s) {
  if (rows < 1 || rows > 0x7fffffffLL || cols < 1 || (!y && (!table || !tokens || vocab < 1)) || (w && !h)) return -1;
  XL_DISPATCH_DTYPE(dtype, T, {
    return cols % 4 == 0 ? launch_rms<T, 4>(x, y, mult, tokens, table, vocab, w, eps, h, rows, cols, s)
                         : launch_rms<T, 1>(x, y, mult, tokens, table, vocab, w, eps, h, rows, cols, s);
  });
  return (int)cudaGetLastError();
}

XL_API int xl_select_rms(const float* x, const int* idx, int stride, int offset, long long x_rows, const float* w, float eps,
                         void* h, int rows, int cols, int dtype, cudaStream_t s) {
  if (rows < 1 || cols < 1 || x_rows < 1 || !w) return -1;
  XL_DISPATCH_DTYPE(dtype, T, {
    select_rms_kernel<T><<<rows, RMS_THREADS, 0, s>>>(x, idx, stride, offset, x_rows, w, eps, (T*)h, cols);
  });
  return (int)cudaGetLastError();
}

// gate: first of 2F columns [gate | up] inside rows of stride ldg; y: first of F columns inside rows of stride ldy.
XL_API int xl_clamped_glu(const void* gate, long long ldg, void* y, long long ldy, long long rows, int F, float limit,
                          float slope, float shift, int dtype, cudaStream_t s) {
  if (rows < 1 || F < 1 || ldg < 2LL * F || ldy < F) return -1;
  XL_DISPATCH_DTYPE(dtype, T, {
    constexpr int V = 16 / sizeof(T);
    if (F % V == 0 && ldg % V == 0 && ldy % V == 0 && (((uintptr_t)gate | (uintptr_t)y) & 15) == 0)
      clamped_glu_kernel<T, V><<<xl_grid_for(rows * (F / V), 256), 256, 0, s>>>((const T*)gate, ldg, (T*)y, ldy, rows, F, limit,
                                                                               slope, shift);
    else
      clamped_glu_kernel<T, 1><<<xl_grid_for(rows * F, 256), 256, 0, s>>>((const T*)gate, ldg, (T*)y, ldy, rows, F, limit,
                                                                         slope, shift);
  });
  return (int)cudaGetLastError();
}

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

// Floats of `pairs` that a portion needs.
XL_API long long xl_min_gru_scratch(int B, int T_len, int W) {
  return 2LL * B * ((T_len + gru_range(T_len) - 1) / gru_range(T_len) + 1) * W;
}

// zxg (B*T_len, 3W) and y (B*T_len, W) of type `dtype`; bz, bx (W), state (B, W), pairs (scratch) fp32; pos, count (B) int32.
// All base pointers 16-byte aligned. Rows of y past count[b] are not written.
XL_API int xl_min_gru(const void* zxg, const float* bz, const float* bx, float* state, void* y, float* pairs, const int* pos,
                      const int* count, int B, int T_len, int W, int dtype, cudaStream_t s) {
  if (B < 1 || B > 65535 || T_len < 1 || W < 1 || !pairs) return -1;
  GruParams p;
  p.bz = bz; p.bx = bx; p.state = state; p.pairs = (float2*)pairs; p.pos = pos; p.count = count; p.T = T_len; p.W = W;
  p.L = gru_range(T_len);
  p.ranges = (T_len + p.L - 1) / p.L + 1;
  XL_DISPATCH_DTYPE(dtype, T, {
    return W % 2 == 0 ? launch_min_gru<T, 2>(zxg, y, p, B, s) : launch_min_gru<T, 1>(zxg, y, p, B, s);
  });
  return (int)cudaGetLastError();
}
