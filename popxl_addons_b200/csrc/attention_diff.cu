// Differential attention against a key / value cache, with chunked visibility.
//
// Every query head holds two query / key maps over the same values. With a_m = softmax(scale * q_m K_m^T) V for map m:
//   o = a_1 - lambda * a_2,   out = o / sqrt(mean(o^2) + eps) * out_scale          (mean over the head's value features)
// Position i attends j <= i; with chunk > 0 only positions of its own chunk (floor(i / chunk) == floor(j / chunk)), so its
// first key is (i / chunk) * chunk. Heads are grouped: query head h reads key / value head h / (H / G).
//
// A portion holds `T` rows per sequence, of which the first count[b] are real, at positions pos[b] ... The new keys (rotated)
// and values go into the caches first, attention then reads everything from there:
//   projections (B*T, ld): [q: H x 2 x dim | k: G x 2 x dim | v: G x vdim]
//   k cache (B, G, 2, Smax, dim), v cache (B, G, Smax, vdim)
//
//   xl_diff_rope_append    rotate q in place, k into the cache, v into the cache
//   xl_diff_attn_general   any sizes and types, scores and weights in fp32 on the CUDA cores: one warp per row and head
//   xl_diff_attn_decode    one token per sequence, bf16: rotation, append, attention and the combination in one launch
#include "attention_decode.cuh"

#include <math.h>

namespace {

// ---- rotary + append -----------------------------------------------------------------------------------------------
// One thread per feature pair of a row's q and k heads, and per two value features. Interleaved pairs (2i, 2i+1), i < R/2.
template <typename T>
__global__ void __launch_bounds__(256)
    diff_rope_append_kernel(T* __restrict__ qkv, long long ld, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                            T* __restrict__ kc, T* __restrict__ vc, const int* __restrict__ pos, const int* __restrict__ count,
                            long long rows, int T_len, int H, int G, int dim, int vdim, int R, int Smax) {
  const int half = (dim + 1) / 2, vhalf = (vdim + 1) / 2;
  const int nq = H * 2 * half, nk = G * 2 * half, nv = G * vhalf;
  const long long per_row = nq + nk + nv, total = rows * per_row;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long row = i / per_row;
    int u = (int)(i - row * per_row);
    const int b = (int)(row / T_len), t = (int)(row - (long long)b * T_len);
    const int p = pos[b] + t;
    if (t >= count[b] || p < 0 || p >= Smax) continue;
    T* src = qkv + row * ld;
    if (u < nq + nk) {
      const bool is_q = u < nq;
      if (!is_q) u -= nq;
      const int hm = u / half, e = (u - hm * half) * 2;
      T* s = src + (is_q ? 0 : (long long)H * 2 * dim) + (long long)hm * dim + e;
      const bool two = e + 1 < dim;
      float x0 = xl_to_float(s[0]), x1 = two ? xl_to_float(s[1]) : 0.f;
      if (e < R) {
        const float c = cos_t[(long long)p * (R / 2) + e / 2], sn = sin_t[(long long)p * (R / 2) + e / 2];
        const float y0 = x0 * c - x1 * sn, y1 = x1 * c + x0 * sn;
        x0 = y0;
        x1 = y1;
        if (is_q) {
          s[0] = xl_from_float<T>(x0);
          if (two) s[1] = xl_from_float<T>(x1);
        }
      }
      if (!is_q) {
        T* d = kc + (((long long)b * G * 2 + hm) * Smax + p) * dim + e;
        d[0] = xl_from_float<T>(x0);
        if (two) d[1] = xl_from_float<T>(x1);
      }
    } else {
      u -= nq + nk;
      const int g = u / vhalf, e = (u - g * vhalf) * 2;
      const T* s = src + (long long)(H + G) * 2 * dim + (long long)g * vdim + e;
      T* d = vc + (((long long)b * G + g) * Smax + p) * vdim + e;
      d[0] = s[0];
      if (e + 1 < vdim) d[1] = s[1];
    }
  }
}

// The same for sizes that are multiples of eight (dim, vdim, R even): eight features per thread through 16-byte accesses.
template <typename T> struct alignas(16) Pack16 { T v[16 / sizeof(T)]; };
template <typename T>
__global__ void __launch_bounds__(256)
    diff_rope_append_vec_kernel(T* __restrict__ qkv, long long ld, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                T* __restrict__ kc, T* __restrict__ vc, const int* __restrict__ pos, const int* __restrict__ count,
                                int T_len, int H, int G, int dim, int vdim, int R, int Smax) {
  constexpr int V = 16 / sizeof(T);
  const int b = blockIdx.y, t = blockIdx.x, p = pos[b] + t;
  if (t >= count[b] || p < 0 || p >= Smax) return;
  T* src = qkv + ((long long)b * T_len + t) * ld;
  const float* cs = cos_t + (long long)p * (R / 2);
  const float* sn = sin_t + (long long)p * (R / 2);
  const int per = dim / V, nq = H * 2 * per, nk = G * 2 * per, per_v = vdim / V, nv = G * per_v;
  for (int u = threadIdx.x; u < nq + nk + nv; u += blockDim.x) {
    if (u < nq + nk) {
      const bool is_q = u < nq;
      const int w = is_q ? u : u - nq, hm = w / per, e = (w - hm * per) * V;
      if (is_q && e >= R) continue;  // passes unchanged, in place
      T* sp = src + (is_q ? 0 : (long long)H * 2 * dim) + (long long)hm * dim + e;
      Pack16<T> x = *reinterpret_cast<const Pack16<T>*>(sp);
#pragma unroll
      for (int i = 0; i < V; i += 2) {
        if (e + i < R) {
          const float c = cs[(e + i) / 2], s = sn[(e + i) / 2], x0 = xl_to_float(x.v[i]), x1 = xl_to_float(x.v[i + 1]);
          x.v[i] = xl_from_float<T>(x0 * c - x1 * s);
          x.v[i + 1] = xl_from_float<T>(x1 * c + x0 * s);
        }
      }
      if (is_q) *reinterpret_cast<Pack16<T>*>(sp) = x;
      else *reinterpret_cast<Pack16<T>*>(kc + (((long long)b * G * 2 + hm) * Smax + p) * dim + e) = x;
    } else {
      const int w = u - nq - nk, g = w / per_v, e = (w - g * per_v) * V;
      *reinterpret_cast<Pack16<T>*>(vc + (((long long)b * G + g) * Smax + p) * vdim + e) =
          *reinterpret_cast<const Pack16<T>*>(src + (long long)(H + G) * 2 * dim + (long long)g * vdim + e);
    }
  }
}

// ---- general kernel --------------------------------------------------------------------------------------------------
constexpr int DG_WARPS = 4;
constexpr int DG_MAX_DIM = 512;   // query / key features per map; value features: 32 per DG_VPL, at most 512

template <typename T, int DG_VPL>
__global__ void __launch_bounds__(DG_WARPS * 32)
    diff_attn_general_kernel(const T* __restrict__ q, long long ldq, const T* __restrict__ kc, const T* __restrict__ vc,
                             T* __restrict__ out, long long ldo, const int* __restrict__ pos, const int* __restrict__ count,
                             const float* __restrict__ lam, int T_len, int H, int G, int dim, int vdim, int Smax, int chunk,
                             float scale, float eps, float out_scale) {
  __shared__ float sq[DG_WARPS][2][DG_MAX_DIM];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z, g = h / (H / G);
  const int t = blockIdx.x * DG_WARPS + warp;
  if (t >= min(count[b], T_len)) return;
  const int p = pos[b] + t;
  if (p < 0 || p >= Smax) return;
  const long long row = (long long)b * T_len + t;
  for (int m = 0; m < 2; ++m)
    for (int d = lane; d < dim; d += 32) sq[warp][m][d] = xl_to_float(q[row * ldq + ((long long)h * 2 + m) * dim + d]);
  __syncwarp();
  const int first = chunk > 0 ? (p / chunk) * chunk : 0;
  float o[2][DG_VPL], mx[2], l[2];
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    mx[m] = -INFINITY;
    l[m] = 0.f;
#pragma unroll
    for (int e = 0; e < DG_VPL; ++e) o[m][e] = 0.f;
  }
  const T* vb = vc + ((long long)b * G + g) * Smax * vdim;
  for (int j0 = first; j0 <= p; j0 += 32) {
    const int j = j0 + lane;
    float w[2];
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      float s = -INFINITY;
      if (j <= p) {
        const T* kr = kc + ((((long long)b * G + g) * 2 + m) * Smax + j) * dim;
        s = 0.f;
        for (int d = 0; d < dim; ++d) s = fmaf(sq[warp][m][d], xl_to_float(kr[d]), s);
        s *= scale;
      }
      const float m_new = fmaxf(mx[m], xl_warp_max(s));  // finite: key j0 is visible
      const float corr = expf(mx[m] - m_new);
      w[m] = expf(s - m_new);
      l[m] = l[m] * corr + xl_warp_sum(w[m]);
      mx[m] = m_new;
#pragma unroll
      for (int e = 0; e < DG_VPL; ++e) o[m][e] *= corr;
    }
    const int n = min(32, p - j0 + 1);
    for (int k = 0; k < n; ++k) {
      const float w0 = __shfl_sync(0xffffffffu, w[0], k), w1 = __shfl_sync(0xffffffffu, w[1], k);
      const T* vr = vb + (long long)(j0 + k) * vdim;
#pragma unroll
      for (int e = 0; e < DG_VPL; ++e) {
        if (lane + 32 * e < vdim) {
          const float v = xl_to_float(vr[lane + 32 * e]);
          o[0][e] = fmaf(w0, v, o[0][e]);
          o[1][e] = fmaf(w1, v, o[1][e]);
        }
      }
    }
  }
  const float lambda = *lam;
  float c[DG_VPL], ss = 0.f;
#pragma unroll
  for (int e = 0; e < DG_VPL; ++e) {
    c[e] = lane + 32 * e < vdim ? o[0][e] / l[0] - lambda * (o[1][e] / l[1]) : 0.f;
    ss += c[e] * c[e];
  }
  ss = xl_warp_sum(ss);
  const float f = out_scale / sqrtf(ss / vdim + eps);
#pragma unroll
  for (int e = 0; e < DG_VPL; ++e)
    if (lane + 32 * e < vdim) out[row * ldo + (long long)h * vdim + lane + 32 * e] = xl_from_float<T>(c[e] * f);
}

// ---- decoding: one query row per sequence ------------------------------------------------------------------------------
// Grid (splits, G * head chunks, B). A CTA takes up to 8 query heads of one key / value head and a range of the visible
// keys; its 4 warps walk 16-key blocks independently, each through a cp.async ring of its own, with online softmax state in
// registers. Products on mma.sync with register operands: the row tile of 16 is [map 1: 8 heads | map 2: 8 heads]; scores are
// Q1 K1^T with map 2's rows zero plus Q2 K2^T with map 1's rows zero, so one accumulator holds both maps, and its layout is
// the operand layout of the second product P V, which both maps share. P enters that product as a sum of two bf16 numbers
// (value and rounding error), so the weights keep more than 16 bits. Slices are merged by the CTA that arrives last.
constexpr int DD_WARPS = 4;
constexpr int DD_KEYS = 16;       // keys per block
constexpr int DD_HEADS = 8;       // query heads per CTA
constexpr int DD_RING_LIMIT = 104 * 1024;
constexpr int DD_MAX_SPLITS = 64;

struct DecodeParams {
  const __nv_bfloat16* qkv;
  long long ld;
  const float *cos_t, *sin_t;
  __nv_bfloat16 *kc, *vc, *out;
  long long ldo;
  const int *pos, *count;
  const float* lam;
  int H, G, dim, vdim, R, Smax, chunk;
  float scale, eps, out_scale;
  float* part;             // [B * G * head chunks][splits][16][vdim + 2]
  unsigned int* counters;  // [B * G * head chunks], zero between launches
  int stages;
};

// bytes of one ring stage of one warp: 16 keys x 2 maps x KD pieces of 64 B, then 16 value rows of vdim + 8 elements
__host__ __device__ constexpr int dd_stage_bytes(int kd, int vdim) { return DD_KEYS * 2 * kd * 64 + DD_KEYS * (vdim + 8) * 2; }

// KD: 32-feature steps of a query / key row (dim <= 32 KD); VT: 8-feature tiles of a value row (vdim <= 8 VT)
template <int KD, int VT>
__global__ void __launch_bounds__(DD_WARPS * 32) diff_attn_decode_kernel(const DecodeParams p) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ __align__(16) __nv_bfloat16 sq[2][DD_HEADS][KD * 32];
  __shared__ float sm[DD_WARPS][16], sl[DD_WARPS][16];
  __shared__ float wt[DD_MAX_SPLITS * 16], wl[DD_MAX_SPLITS * 16];  // maxima, then weights, and sums of the slices
  __shared__ unsigned int is_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quad = lane >> 2, j = lane & 3;
  const int per_g = p.H / p.G, hchunks = (per_g + DD_HEADS - 1) / DD_HEADS;
  const int split = blockIdx.x, splits = gridDim.x, g = blockIdx.y / hchunks, b = blockIdx.z;
  const int h0 = g * per_g + (blockIdx.y % hchunks) * DD_HEADS;  // first query head of this CTA
  const int nh = min(DD_HEADS, (g + 1) * per_g - h0);
  const int pos = p.pos[b];
  if (p.count[b] <= 0 || pos < 0 || pos >= p.Smax) {
    xl_grid_dependency_wait();  // no kernel of a chain ends before its predecessor
    return;
  }
  const int first = p.chunk > 0 ? (pos / p.chunk) * p.chunk : 0;
  const int len = pos + 1 - first;
  const int blocks = (len + DD_KEYS - 1) / DD_KEYS;
  const int blk0 = (int)((long long)split * blocks / splits), blk1 = (int)((long long)(split + 1) * blocks / splits);
  const __nv_bfloat16* row = p.qkv + (long long)b * p.ld;
  const __nv_bfloat16* kb = p.kc + ((long long)b * p.G + g) * 2 * p.Smax * p.dim;
  const __nv_bfloat16* vb = p.vc + ((long long)b * p.G + g) * p.Smax * p.vdim;

  // ---- the ring of key / value blocks: a range without the new key starts to load right away --------------------------------
  const int stage_bytes = dd_stage_bytes(KD, p.vdim), vld = p.vdim + 8;
  uint8_t* ring = smem + (long long)warp * p.stages * stage_bytes;
  const int mine = (blk1 - blk0 - warp + DD_WARPS - 1) / DD_WARPS;  // this warp's blocks: blk0 + warp, + DD_WARPS, ...
  auto prefetch = [&](int n) {
    if (n < mine) {
      uint8_t* st = ring + (n % p.stages) * stage_bytes;
      const int key0 = first + (blk0 + warp + n * DD_WARPS) * DD_KEYS;
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          const int key = min(key0 + t * 8 + quad, pos);  // rows past the end repeat the last one and are masked
          const __nv_bfloat16* src = kb + ((long long)m * p.Smax + key) * p.dim;
#pragma unroll
          for (int i = 0; i < KD; ++i) {
            uint8_t* dst = st + (((m * 2 + t) * KD + i) * 32 + lane) * 16;
            if (i * 32 + j * 8 < p.dim) dd_cp16(dst, src + i * 32 + j * 8);
            else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
          }
        }
      uint8_t* sv = st + DD_KEYS * 2 * KD * 64;
      const int pieces = p.vdim / 8;
      for (int i = lane; i < DD_KEYS * pieces; i += 32) {
        const int k = i / pieces, c = i % pieces;
        dd_cp16(sv + (k * vld + c * 8) * 2, vb + (long long)min(key0 + k, pos) * p.vdim + c * 8);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");  // possibly empty: keeps the group count per block fixed
  };
  const bool appends = split == splits - 1;
  if (!appends)
    for (int n = 0; n < p.stages - 1; ++n) prefetch(n);
  xl_grid_dependency_wait();  // the new projections; positions and older keys were there before the previous kernel started
  xl_grid_launch_dependents();
  // ---- rotated queries to shared memory; the CTAs with the last keys append the new key and value (the same data each) ----
  const int half = p.dim / 2;  // dim is even
  auto rotated = [&](const __nv_bfloat16* s, int e, float& y0, float& y1) {
    const float x0 = __bfloat162float(s[0]), x1 = __bfloat162float(s[1]);
    if (e < p.R) {
      const float c = p.cos_t[(long long)pos * (p.R / 2) + e / 2], sn = p.sin_t[(long long)pos * (p.R / 2) + e / 2];
      y0 = x0 * c - x1 * sn;
      y1 = x1 * c + x0 * sn;
    } else {
      y0 = x0;
      y1 = x1;
    }
  };
  for (int i = threadIdx.x; i < 2 * DD_HEADS * KD * 16; i += blockDim.x) {
    const int e = (i % (KD * 16)) * 2, hm = i / (KD * 16), m = hm / DD_HEADS, r = hm % DD_HEADS;
    float y0 = 0.f, y1 = 0.f;
    if (r < nh && e < p.dim) rotated(row + ((long long)(h0 + r) * 2 + m) * p.dim + e, e, y0, y1);
    *reinterpret_cast<uint32_t*>(&sq[m][r][e]) = dd_pack(y0, y1);
  }
  if (appends) {
    for (int i = threadIdx.x; i < 2 * half; i += blockDim.x) {
      const int m = i / half, e = (i % half) * 2;
      float y0, y1;
      rotated(row + ((long long)(p.H + g) * 2 + m) * p.dim + e, e, y0, y1);
      *reinterpret_cast<uint32_t*>(p.kc + ((((long long)b * p.G + g) * 2 + m) * p.Smax + pos) * p.dim + e) = dd_pack(y0, y1);
    }
    const __nv_bfloat16* vsrc = row + (long long)(p.H + p.G) * 2 * p.dim + (long long)g * p.vdim;
    __nv_bfloat16* vdst = p.vc + (((long long)b * p.G + g) * p.Smax + pos) * p.vdim;
    for (int i = threadIdx.x; i < p.vdim; i += blockDim.x) vdst[i] = vsrc[i];
    __threadfence();
  }
  __syncthreads();
  uint4 q1[KD], q2[KD];
#pragma unroll
  for (int i = 0; i < KD; ++i) {
    q1[i] = *reinterpret_cast<const uint4*>(&sq[0][quad][i * 32 + j * 8]);
    q2[i] = *reinterpret_cast<const uint4*>(&sq[1][quad][i * 32 + j * 8]);
  }
  float o[VT][4];
#pragma unroll
  for (int t = 0; t < VT; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[t][e] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};  // rows quad (map 1) and quad + 8 (map 2)
  const float sc = p.scale * 1.4426950408889634f;
  if (appends)
    for (int n = 0; n < p.stages - 1; ++n) prefetch(n);
  for (int n = 0; n < mine; ++n) {
    prefetch(n + p.stages - 1);
    if (p.stages == 2) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 2;" ::: "memory");
    __syncwarp();
    const uint8_t* st = ring + (n % p.stages) * stage_bytes;
    const int key0 = first + (blk0 + warp + n * DD_WARPS) * DD_KEYS;
    float s[2][4];
#pragma unroll
    for (int t = 0; t < 2; ++t) {
#pragma unroll
      for (int e = 0; e < 4; ++e) s[t][e] = 0.f;
#pragma unroll
      for (int i = 0; i < KD; ++i) {
        const uint4 k1 = *reinterpret_cast<const uint4*>(st + ((t * KD + i) * 32 + lane) * 16);
        const uint4 k2 = *reinterpret_cast<const uint4*>(st + (((2 + t) * KD + i) * 32 + lane) * 16);
        dd_mma(s[t], q1[i].x, 0u, q1[i].y, 0u, k1.x, k1.y);
        dd_mma(s[t], 0u, q2[i].x, 0u, q2[i].y, k2.x, k2.y);
        dd_mma(s[t], q1[i].z, 0u, q1[i].w, 0u, k1.z, k1.w);
        dd_mma(s[t], 0u, q2[i].z, 0u, q2[i].w, k2.z, k2.w);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e)
        s[t][e] = key0 + t * 8 + 2 * j + (e & 1) <= pos ? s[t][e] * sc : -INFINITY;
    }
    float alpha[2];
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      float v = fmaxf(fmaxf(s[0][2 * m], s[0][2 * m + 1]), fmaxf(s[1][2 * m], s[1][2 * m + 1]));
      v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
      v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
      const float m_new = fmaxf(mx[m], v);  // finite: the first key of a block is always visible
      alpha[m] = exp2f(mx[m] - m_new);
      mx[m] = m_new;
      float sum = 0.f;
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          s[t][2 * m + e] = exp2f(s[t][2 * m + e] - m_new);
          sum += s[t][2 * m + e];
        }
      l[m] = l[m] * alpha[m] + sum;  // this lane's share of the row sum
    }
    uint32_t ph[4], pl[4];
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const float x = s[t][2 * m], y = s[t][2 * m + 1];
        const uint32_t hi = dd_pack(x, y);
        ph[2 * t + m] = hi;
        pl[2 * t + m] = dd_pack(x - dd_lo(hi), y - dd_hi(hi));
      }
    const uint32_t sv = (uint32_t)__cvta_generic_to_shared(st + DD_KEYS * 2 * KD * 64);
    const uint32_t vaddr = sv + (((lane & 7) + ((lane >> 3) & 1) * 8) * vld + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int t = 0; t < VT; t += 2) {
      if (t * 8 < p.vdim) {
        uint32_t v0, v1, v2, v3;  // key pairs of value tiles t (v0, v1) and t + 1 (v2, v3)
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                     : "=r"(v0), "=r"(v1), "=r"(v2), "=r"(v3)
                     : "r"(vaddr + t * 16));
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          o[t + u][0] *= alpha[0];
          o[t + u][1] *= alpha[0];
          o[t + u][2] *= alpha[1];
          o[t + u][3] *= alpha[1];
        }
        dd_mma(o[t], ph[0], ph[1], ph[2], ph[3], v0, v1);
        dd_mma(o[t + 1], ph[0], ph[1], ph[2], ph[3], v2, v3);
        dd_mma(o[t], pl[0], pl[1], pl[2], pl[3], v0, v1);
        dd_mma(o[t + 1], pl[0], pl[1], pl[2], pl[3], v2, v3);
      }
    }
    __syncwarp();  // every lane has read the stage before it is refilled
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    l[m] += __shfl_xor_sync(0xffffffffu, l[m], 1);
    l[m] += __shfl_xor_sync(0xffffffffu, l[m], 2);
    if (j == 0) {
      sm[warp][quad + 8 * m] = mx[m];
      sl[warp][quad + 8 * m] = l[m];
    }
  }
  __syncthreads();  // all rings are idle: their memory holds the warps' outputs from here on
  float* so = reinterpret_cast<float*>(smem);  // [DD_WARPS][16][vdim]
#pragma unroll
  for (int t = 0; t < VT; ++t) {
    if (t * 8 < p.vdim) {
      float* d = so + ((long long)warp * 16 + quad) * p.vdim + t * 8 + 2 * j;
      d[0] = o[t][0];
      d[1] = o[t][1];
      d += 8 * p.vdim;
      d[0] = o[t][2];
      d[1] = o[t][3];
    }
  }
  __syncthreads();
  // ---- merge of the warps; the slice's result goes to `part`, or stays here when there is one slice ------------------------
  __shared__ float fm[16], fl[16];
  const long long unit = (long long)b * gridDim.y + blockIdx.y;
  const int pw = p.vdim + 2;
  float* mypart = p.part + (unit * splits + split) * 16 * pw;
  if (threadIdx.x < 16) {
    const int r = threadIdx.x;
    float m = -INFINITY, ll = 0.f;
    for (int w = 0; w < DD_WARPS; ++w) m = fmaxf(m, sm[w][r]);
    for (int w = 0; w < DD_WARPS; ++w) ll += sm[w][r] == -INFINITY ? 0.f : sl[w][r] * exp2f(sm[w][r] - m);
    fm[r] = m;
    fl[r] = ll;
    if (splits > 1) {
      __stcg(mypart + r * pw, m);
      __stcg(mypart + r * pw + 1, ll);
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < 2 * nh * p.vdim; i += blockDim.x) {
    const int rr = i / p.vdim, c = i - rr * p.vdim, r = rr < nh ? rr : DD_HEADS + rr - nh;  // rows in use
    float acc = 0.f;
#pragma unroll
    for (int w = 0; w < DD_WARPS; ++w)
      acc += sm[w][r] == -INFINITY ? 0.f : so[((long long)w * 16 + r) * p.vdim + c] * exp2f(sm[w][r] - fm[r]);
    if (splits > 1) __stcg(mypart + r * pw + 2 + c, acc);
    else so[(long long)r * p.vdim + c] = acc;  // warp 0's copy: read and written by this thread only
  }
  if (splits > 1) {
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) is_last = atomicAdd(p.counters + unit, 1u) == (unsigned int)splits - 1;
    __syncthreads();
    if (!is_last) return;
    __threadfence();
    const float* parts = p.part + unit * splits * 16 * pw;
    for (int i = threadIdx.x; i < splits * 16; i += blockDim.x) {
      wt[i] = __ldcg(parts + (long long)i * pw);
      wl[i] = __ldcg(parts + (long long)i * pw + 1);
    }
    __syncthreads();
    if (threadIdx.x < 16) {
      float m = -INFINITY, ll = 0.f;
      for (int k = 0; k < splits; ++k) m = fmaxf(m, wt[k * 16 + threadIdx.x]);
      for (int k = 0; k < splits; ++k) {
        float& w = wt[k * 16 + threadIdx.x];
        w = w == -INFINITY ? 0.f : exp2f(w - m);
        ll += w * wl[k * 16 + threadIdx.x];
      }
      fl[threadIdx.x] = ll;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < 2 * nh * p.vdim; i += blockDim.x) {
      const int rr = i / p.vdim, c = i - rr * p.vdim, r = rr < nh ? rr : DD_HEADS + rr - nh;
      const float* src = parts + (long long)r * pw + 2 + c;
      float acc = 0.f;
#pragma unroll 8
      for (int k = 0; k < splits; ++k) acc += wt[k * 16 + r] * __ldcg(src + (long long)k * 16 * pw);
      so[(long long)r * p.vdim + c] = acc;
    }
    if (threadIdx.x == 0) p.counters[unit] = 0;
  }
  __syncthreads();
  // ---- a_1 - lambda a_2, divided by its root mean square: one warp per head -------------------------------------------------
  const float lambda = *p.lam;
  for (int r = warp; r < nh; r += DD_WARPS) {
    const float i1 = 1.f / fl[r], i2 = lambda / fl[r + 8];
    float ss = 0.f;
    for (int c = lane; c < p.vdim; c += 32) {
      const float v = so[(long long)r * p.vdim + c] * i1 - so[(long long)(r + 8) * p.vdim + c] * i2;
      so[(long long)r * p.vdim + c] = v;
      ss += v * v;
    }
    ss = xl_warp_sum(ss);
    const float f = p.out_scale / sqrtf(ss / p.vdim + p.eps);
    for (int c = lane; c < p.vdim; c += 32)
      p.out[(long long)b * p.ldo + (long long)(h0 + r) * p.vdim + c] = __float2bfloat16_rn(so[(long long)r * p.vdim + c] * f);
  }
}

template <int KD, int VT> int dd_launch(DecodeParams p, int B, int splits, cudaStream_t s) {
  const int stage = dd_stage_bytes(KD, p.vdim) * DD_WARPS;
  p.stages = 3 * stage <= DD_RING_LIMIT ? 3 : 2;
  int bytes = p.stages * stage;
  const int merge = DD_WARPS * 16 * p.vdim * 4;
  if (bytes < merge) bytes = merge;
  static int configured = 0;
  if (configured < bytes) {
    const cudaError_t e = cudaFuncSetAttribute(diff_attn_decode_kernel<KD, VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return (int)e;
    configured = bytes;
  }
  const int hchunks = (p.H / p.G + DD_HEADS - 1) / DD_HEADS;
  const cudaError_t e = xl_launch_overlapped(diff_attn_decode_kernel<KD, VT>, dim3(splits, p.G * hchunks, B), dim3(DD_WARPS * 32),
                                             (size_t)bytes, s, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

}  // namespace

// qkv: (B*T_len, ld) as described above, q rotated in place. cos / sin tables (Smax, R/2) fp32 (null when R == 0).
XL_API int xl_diff_rope_append(void* qkv, long long ld, const float* cos_t, const float* sin_t, void* kc, void* vc,
                               const int* pos, const int* count, int B, int T_len, int H, int G, int dim, int vdim, int R,
                               int Smax, int dtype, cudaStream_t s) {
  if (B < 1 || T_len < 1 || G < 1 || H % G || dim < 1 || vdim < 1 || R < 0 || R > dim || (R & 1) || Smax < 1) return -1;
  if (R > 0 && (!cos_t || !sin_t)) return -1;
  const long long rows = (long long)B * T_len;
  const long long items = rows * ((long long)(H + G) * 2 * ((dim + 1) / 2) + (long long)G * ((vdim + 1) / 2));
  if (dim % 8 == 0 && vdim % 8 == 0 && ld % 8 == 0 && B <= 65535 && ((uintptr_t)qkv & 15) == 0 && ((uintptr_t)kc & 15) == 0 &&
      ((uintptr_t)vc & 15) == 0) {
    XL_DISPATCH_DTYPE(dtype, T, {
      diff_rope_append_vec_kernel<T><<<dim3(T_len, B), 256, 0, s>>>((T*)qkv, ld, cos_t, sin_t, (T*)kc, (T*)vc, pos, count, T_len,
                                                                   H, G, dim, vdim, R, Smax);
    });
    return (int)cudaGetLastError();
  }
  XL_DISPATCH_DTYPE(dtype, T, {
    diff_rope_append_kernel<T><<<xl_grid_for(items, 256), 256, 0, s>>>((T*)qkv, ld, cos_t, sin_t, (T*)kc, (T*)vc, pos, count,
                                                                      rows, T_len, H, G, dim, vdim, R, Smax);
  });
  return (int)cudaGetLastError();
}

// q: (B*T_len, ldq), rotated; out: (B*T_len, ldo). dim <= 512, vdim <= 512. chunk 0: plain causal. Rows past count[b] of a
// sequence are left as they are.
XL_API int xl_diff_attn_general(const void* q, long long ldq, const void* kc, const void* vc, void* out, long long ldo,
                                const int* pos, const int* count, const float* lam, int B, int T_len, int H, int G, int dim,
                                int vdim, int Smax, int chunk, float scale, float eps, float out_scale, int dtype,
                                cudaStream_t s) {
  if (B < 1 || B > 65535 || H < 1 || H > 65535 || T_len < 1 || G < 1 || H % G || dim < 1 || dim > DG_MAX_DIM || vdim < 1 ||
      vdim > 512 || Smax < 1 || chunk < 0)
    return -1;
  const dim3 grid((T_len + DG_WARPS - 1) / DG_WARPS, H, B);
  XL_DISPATCH_DTYPE(dtype, T, {
    if (vdim <= 256)
      diff_attn_general_kernel<T, 8><<<grid, DG_WARPS * 32, 0, s>>>((const T*)q, ldq, (const T*)kc, (const T*)vc, (T*)out, ldo,
                                                                   pos, count, lam, T_len, H, G, dim, vdim, Smax, chunk, scale,
                                                                   eps, out_scale);
    else
      diff_attn_general_kernel<T, 16><<<grid, DG_WARPS * 32, 0, s>>>((const T*)q, ldq, (const T*)kc, (const T*)vc, (T*)out, ldo,
                                                                    pos, count, lam, T_len, H, G, dim, vdim, Smax, chunk, scale,
                                                                    eps, out_scale);
  });
  return (int)cudaGetLastError();
}

// One token per sequence (rows of qkv = sequences), bf16. dim, vdim multiples of 8, dim <= 128, vdim <= 256, ld a multiple of
// 8. The new key and value are rotated / appended by the kernel; q is not modified. part: B * G * ceil(H/G/8) * splits * 16 *
// (vdim + 2) floats; counters: B * G * ceil(H/G/8) zero-initialised words (left zeroed). Sequences with count 0 are skipped.
XL_API int xl_diff_attn_decode(const void* qkv, long long ld, const float* cos_t, const float* sin_t, void* kc, void* vc,
                               void* out, long long ldo, const int* pos, const int* count, const float* lam, int B, int H, int G,
                               int dim, int vdim, int R, int Smax, int chunk, float scale, float eps, float out_scale,
                               int splits, float* part, unsigned int* counters, cudaStream_t s) {
  if (B < 1 || B > 65535 || G < 1 || H % G || H > 4096 || dim < 8 || dim > 128 || dim % 8 || vdim < 8 || vdim > 256 || vdim % 8 ||
      R < 0 || R > dim || (R & 1) || Smax < 1 || chunk < 0 || splits < 1 || splits > DD_MAX_SPLITS || (ld % 8))
    return -1;
  if (((uintptr_t)qkv & 15) || ((uintptr_t)kc & 15) || ((uintptr_t)vc & 15) || (R > 0 && (!cos_t || !sin_t))) return -1;
  if (splits > 1 && (!part || !counters)) return -1;
  DecodeParams p = {};
  p.qkv = (const __nv_bfloat16*)qkv; p.ld = ld; p.cos_t = cos_t; p.sin_t = sin_t;
  p.kc = (__nv_bfloat16*)kc; p.vc = (__nv_bfloat16*)vc; p.out = (__nv_bfloat16*)out; p.ldo = ldo;
  p.pos = pos; p.count = count; p.lam = lam; p.H = H; p.G = G; p.dim = dim; p.vdim = vdim; p.R = R; p.Smax = Smax;
  p.chunk = chunk; p.scale = scale; p.eps = eps; p.out_scale = out_scale; p.part = part; p.counters = counters;
#define XL_DD(KD)                                       \
  if (vdim <= 64) return dd_launch<KD, 8>(p, B, splits, s);   \
  if (vdim <= 128) return dd_launch<KD, 16>(p, B, splits, s); \
  return dd_launch<KD, 32>(p, B, splits, s);
  if (dim <= 32) { XL_DD(1) }
  if (dim <= 64) { XL_DD(2) }
  XL_DD(4)
#undef XL_DD
}
