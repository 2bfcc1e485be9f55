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
#include "common.cuh"

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

// ---- general kernel --------------------------------------------------------------------------------------------------
constexpr int DG_WARPS = 4;
constexpr int DG_MAX_DIM = 256;   // query / key features per map
constexpr int DG_VPL = 8;         // value features per lane: vdim <= 256

template <typename T>
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

}  // namespace

// qkv: (B*T_len, ld) as described above, q rotated in place. cos / sin tables (Smax, R/2) fp32 (null when R == 0).
XL_API int xl_diff_rope_append(void* qkv, long long ld, const float* cos_t, const float* sin_t, void* kc, void* vc,
                               const int* pos, const int* count, int B, int T_len, int H, int G, int dim, int vdim, int R,
                               int Smax, int dtype, cudaStream_t s) {
  if (B < 1 || T_len < 1 || G < 1 || H % G || dim < 1 || vdim < 1 || R < 0 || R > dim || (R & 1) || Smax < 1) return -1;
  if (R > 0 && (!cos_t || !sin_t)) return -1;
  const long long rows = (long long)B * T_len;
  const long long items = rows * ((long long)(H + G) * 2 * ((dim + 1) / 2) + (long long)G * ((vdim + 1) / 2));
  XL_DISPATCH_DTYPE(dtype, T, {
    diff_rope_append_kernel<T><<<xl_grid_for(items, 256), 256, 0, s>>>((T*)qkv, ld, cos_t, sin_t, (T*)kc, (T*)vc, pos, count,
                                                                      rows, T_len, H, G, dim, vdim, R, Smax);
  });
  return (int)cudaGetLastError();
}

// q: (B*T_len, ldq), rotated; out: (B*T_len, ldo). dim <= 256, vdim <= 256. chunk 0: plain causal. Rows past count[b] of a
// sequence are left as they are.
XL_API int xl_diff_attn_general(const void* q, long long ldq, const void* kc, const void* vc, void* out, long long ldo,
                                const int* pos, const int* count, const float* lam, int B, int T_len, int H, int G, int dim,
                                int vdim, int Smax, int chunk, float scale, float eps, float out_scale, int dtype,
                                cudaStream_t s) {
  if (B < 1 || B > 65535 || H < 1 || H > 65535 || T_len < 1 || G < 1 || H % G || dim < 1 || dim > DG_MAX_DIM || vdim < 1 ||
      vdim > 32 * DG_VPL || Smax < 1 || chunk < 0)
    return -1;
  const dim3 grid((T_len + DG_WARPS - 1) / DG_WARPS, H, B);
  XL_DISPATCH_DTYPE(dtype, T, {
    diff_attn_general_kernel<T><<<grid, DG_WARPS * 32, 0, s>>>((const T*)q, ldq, (const T*)kc, (const T*)vc, (T*)out, ldo, pos,
                                                              count, lam, T_len, H, G, dim, vdim, Smax, chunk, scale, eps,
                                                              out_scale);
  });
  return (int)cudaGetLastError();
}
