// Sliding-window attention against a key / value cache: normalised queries and keys, kept first tokens, a sink, a gate.
//
//   q' = q / rms(q) * wq,  k' = k / rms(k) * wk          (per head, over its features)
//   p_j = exp(s_j) / (exp(sink) + sum_j' exp(s_j'))      with s_j = scale * q'.k'_j over the visible j (attention_window.cuh)
//   out = (sum_j p_j v_j) * sigmoid(gate)                 (sink -inf: none; the gate may be absent)
//
// Heads are grouped: query head h reads key / value head h / R with R = H / G. A portion holds `T` rows per sequence, of which
// the first count[b] are real, at positions pos[b] ... New keys and values go into the caches first, attention then reads
// everything from there:
//   projections (B*T, ld): [q: H x dim | k: G x dim | v: G x vdim | gate: H x vdim]
//   k cache (B, G, Smax, dim), v cache (B, G, Smax, vdim)
//   q' (B, G, T, R, dim): the rows that read one key / value head are consecutive, so that a tile can hold several heads
//
//   xl_qk_norm_append        q' to its buffer, k' and v into the caches
//   xl_window_attn_general   any sizes and types, scores and weights in fp32 on the CUDA cores: one warp per row and head
//   xl_window_attn_decode    one token per sequence, bf16: norms, append, attention and gate in one launch
#include "attention_decode.cuh"
#include "attention_window.cuh"

#include <math.h>

namespace {

constexpr int WA_MAX_DIM = 512;

__device__ __forceinline__ float gate_factor(float g) { return 1.f / (1.f + expf(-g)); }

// ---- norms + append ----------------------------------------------------------------------------------------------------
// One CTA per row; `group` lanes (a power of two) share a head. Accesses of V elements, 16 V at most per lane.
template <typename T, int V> struct alignas(V * sizeof(T)) Piece { T v[V]; };

template <typename T, int V>
__global__ void __launch_bounds__(256)
    qk_norm_append_kernel(const T* __restrict__ proj, long long ld, const float* __restrict__ wq, const float* __restrict__ wk,
                          T* __restrict__ qn, T* __restrict__ kc, T* __restrict__ vc, const int* __restrict__ pos,
                          const int* __restrict__ count, int T_len, int H, int G, int dim, int vdim, int Smax, float eps,
                          int group) {
  constexpr int NP = 16 / V;  // pieces per lane: 32 lanes cover WA_MAX_DIM features
  const int b = blockIdx.y, t = blockIdx.x, p = pos[b] + t;
  if (t >= count[b] || p < 0 || p >= Smax) return;
  const T* row = proj + ((long long)b * T_len + t) * ld;
  const int R = H / G, l = threadIdx.x & (group - 1), pieces = dim / V;
  const int heads_at_once = blockDim.x / group;
  for (int h0 = 0; h0 < H + G; h0 += heads_at_once) {
    const int h = h0 + threadIdx.x / group;
    const bool on = h < H + G;
    float x[NP][V], sq = 0.f;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int c = l + i * group;
      if (on && c < pieces) {
        const Piece<T, V> r = *reinterpret_cast<const Piece<T, V>*>(row + (long long)h * dim + c * V);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          x[i][e] = xl_to_float(r.v[e]);
          sq += x[i][e] * x[i][e];
        }
      }
    }
    for (int o = group / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    if (!on) continue;
    const float f = 1.f / sqrtf(sq / dim + eps);
    const bool is_q = h < H;
    const float* w = is_q ? wq : wk;
    T* dst = is_q ? qn + ((((long long)b * G + h / R) * T_len + t) * R + h % R) * dim
                  : kc + (((long long)b * G + (h - H)) * Smax + p) * dim;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int c = l + i * group;
      if (c < pieces) {
        Piece<T, V> r;
#pragma unroll
        for (int e = 0; e < V; ++e) r.v[e] = xl_from_float<T>(x[i][e] * f * w[c * V + e]);
        *reinterpret_cast<Piece<T, V>*>(dst + c * V) = r;
      }
    }
  }
  const T* src = row + (long long)(H + G) * dim;
  const int per_v = vdim / V;
  for (int i = threadIdx.x; i < G * per_v; i += blockDim.x) {
    const int g = i / per_v, c = i - g * per_v;
    *reinterpret_cast<Piece<T, V>*>(vc + (((long long)b * G + g) * Smax + p) * vdim + c * V) =
        *reinterpret_cast<const Piece<T, V>*>(src + (long long)g * vdim + c * V);
  }
}

template <typename T, int V>
int launch_append(const void* proj, long long ld, const float* wq, const float* wk, void* qn, void* kc, void* vc, const int* pos,
                  const int* count, int B, int T_len, int H, int G, int dim, int vdim, int Smax, float eps, cudaStream_t s) {
  int group = 1;
  while (group < 32 && group * V < dim) group *= 2;
  qk_norm_append_kernel<T, V><<<dim3(T_len, B), 256, 0, s>>>((const T*)proj, ld, wq, wk, (T*)qn, (T*)kc, (T*)vc, pos, count, T_len,
                                                             H, G, dim, vdim, Smax, eps, group);
  return (int)cudaGetLastError();
}

// ---- general kernel --------------------------------------------------------------------------------------------------
constexpr int WG_WARPS = 4;

template <typename T, int VPL>  // VPL: value features per lane
__global__ void __launch_bounds__(WG_WARPS * 32)
    window_attn_general_kernel(const T* __restrict__ qn, const T* __restrict__ kc, const T* __restrict__ vc,
                               const T* __restrict__ gate, long long ldg, T* __restrict__ out, long long ldo,
                               const int* __restrict__ pos, const int* __restrict__ count, int T_len, int H, int G, int dim,
                               int vdim, int Smax, int window, int keep_first, float scale, float sink) {
  __shared__ float sq[WG_WARPS][WA_MAX_DIM];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z, R = H / G, g = h / R;
  const int t = blockIdx.x * WG_WARPS + warp;
  if (t >= min(count[b], T_len)) return;
  const int p = pos[b] + t;
  if (p < 0 || p >= Smax) return;
  const T* q = qn + ((((long long)b * G + g) * T_len + t) * R + h % R) * dim;
  for (int d = lane; d < dim; d += 32) sq[warp][d] = xl_to_float(q[d]);
  __syncwarp();
  const WindowRange seen = window_range(p, window, keep_first);
  const T* kb = kc + ((long long)b * G + g) * Smax * dim;
  const T* vb = vc + ((long long)b * G + g) * Smax * vdim;
  float o[VPL], mx = sink, l = sink == -INFINITY ? 0.f : 1.f;
#pragma unroll
  for (int e = 0; e < VPL; ++e) o[e] = 0.f;
  auto walk = [&](int begin, int end) {
    for (int j0 = begin; j0 < end; j0 += 32) {
      const int j = j0 + lane;
      float s = -INFINITY;
      if (j < end) {
        const T* kr = kb + (long long)j * dim;
        s = 0.f;
        for (int d = 0; d < dim; ++d) s = fmaf(sq[warp][d], xl_to_float(kr[d]), s);
        s *= scale;
      }
      const float m_new = fmaxf(mx, xl_warp_max(s));  // finite: key j0 is visible
      const float corr = expf(mx - m_new), w = expf(s - m_new);
      l = l * corr + xl_warp_sum(w);
      mx = m_new;
#pragma unroll
      for (int e = 0; e < VPL; ++e) o[e] *= corr;
      const int n = min(32, end - j0);
      for (int k = 0; k < n; ++k) {
        const float wk = __shfl_sync(0xffffffffu, w, k);
        const T* vr = vb + (long long)(j0 + k) * vdim;
#pragma unroll
        for (int e = 0; e < VPL; ++e)
          if (lane + 32 * e < vdim) o[e] = fmaf(wk, xl_to_float(vr[lane + 32 * e]), o[e]);
      }
    }
  };
  walk(0, seen.kept);
  walk(seen.first, p + 1);
  const long long row = (long long)b * T_len + t;
  const T* gr = gate ? gate + row * ldg + (long long)h * vdim : nullptr;
#pragma unroll
  for (int e = 0; e < VPL; ++e) {
    const int c = lane + 32 * e;
    if (c < vdim) {
      float v = o[e] / l;
      if (gr) v *= gate_factor(xl_to_float(gr[c]));
      out[row * ldo + (long long)h * vdim + c] = xl_from_float<T>(v);
    }
  }
}

// ---- decoding: one query row per sequence ------------------------------------------------------------------------------
// Grid (splits, G * head chunks, B). A CTA takes up to 8 RT query heads of one key / value head and a range of the visible key
// blocks (16 or 32 keys each: those of the kept first tokens, then those of the window); its 4 warps walk their blocks independently,
// each through a cp.async ring of its own, with online softmax state in registers. Products on mma.sync with register
// operands: the rows of the tile are the query heads (RT = 1: the upper eight rows are zero and cost nothing but the MMA), and
// the layout of the scores' accumulator is the operand layout of the second product. The weights enter that product as sums of
// two bf16 numbers (value and rounding error). Slices are merged by the CTA that arrives last, which also adds the sink.
//
// The older keys do not depend on the previous kernel, so every ring starts to load before the kernel waits for it. The new
// key and value reach the caches and, in shared memory, the block they belong to.
constexpr int WD_WARPS = 4;
constexpr int WD_MAX_SPLITS = 64;

struct WindowDecodeParams {
  const __nv_bfloat16* proj;
  long long ld;
  const float *wq, *wk;
  __nv_bfloat16 *kc, *vc, *out;
  long long ldo;
  const int *pos, *count;
  int H, G, dim, vdim, Smax, window, keep_first, gated;
  float scale, sink, eps;
  float* part;             // [B * G * head chunks][splits][heads per CTA][vdim + 2]
  unsigned int* counters;  // [B * G * head chunks], zero between launches
  int stages;
};

// keys per block: more of them where their rows are short, so that the work per block stays about the same
__host__ __device__ constexpr int wd_keys(int kd, int vt) { return 4 * kd + vt <= 16 ? 32 : 16; }
// bytes of one ring stage of one warp: the keys as KD pieces of 64 B, then the value rows of vdim + 8 elements
__host__ __device__ constexpr int wd_stage_bytes(int keys, int kd, int vdim) { return keys * kd * 64 + keys * (vdim + 8) * 2; }

// c += a b for a 16 x 8 tile of which 8 RT rows are in use; a_lo / a_hi: rows quad and quad + 8, two k pairs each.
__device__ __forceinline__ void wd_mma(float (&c)[4], const uint2& a_lo, const uint2& a_hi, uint32_t b0, uint32_t b1) {
  dd_mma(c, a_lo.x, a_hi.x, a_lo.y, a_hi.y, b0, b1);
}
__device__ __forceinline__ void wd_mma(float (&c)[2], const uint2& a_lo, const uint2&, uint32_t b0, uint32_t b1) {
  float unused0, unused1;
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%10,%11,%12,%12};"
               : "=f"(c[0]), "=f"(c[1]), "=f"(unused0), "=f"(unused1)
               : "r"(a_lo.x), "r"(0u), "r"(a_lo.y), "r"(0u), "r"(b0), "r"(b1), "f"(c[0]), "f"(c[1]), "f"(0.f));
}

// KD: 32-feature steps of a query / key row (dim <= 32 KD); VT: 8-feature tiles of a value row (vdim <= 8 VT)
template <int KD, int VT, int RT>
__global__ void __launch_bounds__(WD_WARPS * 32) window_attn_decode_kernel(const WindowDecodeParams p) {
  constexpr int KEYS = wd_keys(KD, VT), KT = KEYS / 8;  // keys per block, tiles of eight keys
  constexpr int HEADS = 8 * RT;
  constexpr int NORMS = HEADS / WD_WARPS + 1;  // query heads per warp, and the new key
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ __align__(16) __nv_bfloat16 sq[HEADS + 1][KD * 32];  // normalised queries; the last row is the new key
  __shared__ float sm[WD_WARPS][HEADS], sl[WD_WARPS][HEADS];
  __shared__ float wt[WD_MAX_SPLITS * HEADS], wl[WD_MAX_SPLITS * HEADS];  // maxima, then weights, and sums of the slices
  __shared__ unsigned int is_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quad = lane >> 2, j = lane & 3;
  const int per_g = p.H / p.G, hchunks = (per_g + HEADS - 1) / HEADS;
  const int split = blockIdx.x, splits = gridDim.x, g = blockIdx.y / hchunks, b = blockIdx.z;
  const int h0 = g * per_g + (blockIdx.y % hchunks) * HEADS;  // first query head of this CTA
  const int nh = min(HEADS, (g + 1) * per_g - h0);
  const int pos = p.pos[b];
  if (p.count[b] <= 0 || pos < 0 || pos >= p.Smax) {
    xl_grid_dependency_wait();  // no kernel of a chain ends before its predecessor
    return;
  }
  const WindowRange seen = window_range(pos, p.window, p.keep_first);
  const int kept_blocks = (seen.kept + KEYS - 1) / KEYS;
  const int blocks = kept_blocks + (pos - seen.first) / KEYS + 1;
  const int blk0 = (int)((long long)split * blocks / splits), blk1 = (int)((long long)(split + 1) * blocks / splits);
  const __nv_bfloat16* row = p.proj + (long long)b * p.ld;
  const __nv_bfloat16* kb = p.kc + ((long long)b * p.G + g) * p.Smax * p.dim;
  const __nv_bfloat16* vb = p.vc + ((long long)b * p.G + g) * p.Smax * p.vdim;
  auto first_key = [&](int blk) { return blk < kept_blocks ? blk * KEYS : seen.first + (blk - kept_blocks) * KEYS; };
  // visible keys of a block lie below this; so do those that are in the cache already, except the new one
  auto end_key = [&](int blk) { return blk < kept_blocks ? seen.kept : pos + 1; };

  // ---- the ring of key / value blocks -------------------------------------------------------------------------------------
  const int stage_bytes = wd_stage_bytes(KEYS, KD, p.vdim), vld = p.vdim + 8;
  uint8_t* ring = smem + (long long)warp * p.stages * stage_bytes;
  const int mine = (blk1 - blk0 - warp + WD_WARPS - 1) / WD_WARPS;  // this warp's blocks: blk0 + warp, + WD_WARPS, ...
  constexpr int V_ROWS = 32 / VT, V_PASSES = KEYS / V_ROWS;  // value rows that a warp copies at a time, one piece per lane
  const int v_row = lane / VT, v_col = (lane % VT) * 8;
  const bool v_on = v_col < p.vdim;
  auto prefetch = [&](int n) {
    if (n < mine) {
      uint8_t* st = ring + (n % p.stages) * stage_bytes;
      const int blk = blk0 + warp + n * WD_WARPS, key0 = first_key(blk), end = min(end_key(blk), pos);
      const bool full = key0 + KEYS <= end;  // else rows from `end` on are zero-filled
#pragma unroll
      for (int t = 0; t < KT; ++t) {
        const bool row_on = full || key0 + t * 8 + quad < end;
        const __nv_bfloat16* src = kb + (row_on ? (long long)(key0 + t * 8 + quad) * p.dim + j * 8 : 0);
#pragma unroll
        for (int i = 0; i < KD; ++i) {
          const bool on = row_on && i * 32 + j * 8 < p.dim;
          dd_cp16_zfill(st + ((t * KD + i) * 32 + lane) * 16, on ? src + i * 32 : kb, on);
        }
      }
      if (v_on) {
        uint8_t* dst = st + KEYS * KD * 64 + (v_row * vld + v_col) * 2;
        const __nv_bfloat16* src = vb + (long long)(key0 + v_row) * p.vdim + v_col;
#pragma unroll
        for (int i = 0; i < V_PASSES; ++i) {
          const bool on = full || key0 + v_row + i * V_ROWS < end;
          dd_cp16_zfill(dst + i * V_ROWS * vld * 2, on ? src + i * V_ROWS * p.vdim : vb, on);
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");  // possibly empty: keeps the group count per block fixed
  };
  for (int n = 0; n < p.stages - 1; ++n) prefetch(n);
  xl_grid_dependency_wait();  // the new projections; positions and older keys were there before the previous kernel started
  xl_grid_launch_dependents();
  // ---- normalised queries and new key to shared memory; the CTAs with the last keys append (the same data each) ---------------
  const bool appends = split == splits - 1;
  const __nv_bfloat16* v_new = row + (long long)(p.H + p.G) * p.dim + (long long)g * p.vdim;
  {
    uint32_t raw[NORMS][2];  // dim <= 128
#pragma unroll
    for (int i = 0; i < NORMS; ++i) {
      const int r = warp + i * WD_WARPS;
      const __nv_bfloat16* src = row + (long long)(r < HEADS ? h0 + r : p.H + g) * p.dim;
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int e = 2 * lane + 64 * u;
        raw[i][u] = (r < nh || r == HEADS) && e < p.dim ? *reinterpret_cast<const uint32_t*>(src + e) : 0u;
      }
    }
    float w[2][4];  // query and key factors
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int e = 2 * lane + 64 * u;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        w[0][2 * u + c] = e < p.dim ? p.wq[e + c] : 0.f;
        w[1][2 * u + c] = e < p.dim ? p.wk[e + c] : 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < NORMS; ++i) {
      const int r = warp + i * WD_WARPS;
      if (r > HEADS) break;
      float x[4], sum = 0.f;
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        x[2 * u] = dd_lo(raw[i][u]);
        x[2 * u + 1] = dd_hi(raw[i][u]);
        sum += x[2 * u] * x[2 * u] + x[2 * u + 1] * x[2 * u + 1];
      }
      const float f = 1.f / sqrtf(xl_warp_sum(sum) / p.dim + p.eps);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int e = 2 * lane + 64 * u;
        if (e < KD * 32) {
          const float w0 = r == HEADS ? w[1][2 * u] : w[0][2 * u], w1 = r == HEADS ? w[1][2 * u + 1] : w[0][2 * u + 1];
          const uint32_t y = dd_pack(x[2 * u] * f * w0, x[2 * u + 1] * f * w1);
          *reinterpret_cast<uint32_t*>(&sq[r][e]) = y;  // rows and features that are not in use: zero
          if (r == HEADS && appends && e < p.dim)
            *reinterpret_cast<uint32_t*>(p.kc + (((long long)b * p.G + g) * p.Smax + pos) * p.dim + e) = y;
        }
      }
    }
    if (appends) {
      __nv_bfloat16* vdst = p.vc + (((long long)b * p.G + g) * p.Smax + pos) * p.vdim;
      for (int i = threadIdx.x; i < p.vdim / 8; i += blockDim.x)
        *reinterpret_cast<uint4*>(vdst + i * 8) = *reinterpret_cast<const uint4*>(v_new + i * 8);
    }
  }
  __syncthreads();
  uint4 q[RT][KD];  // rows quad (and quad + 8)
#pragma unroll
  for (int m = 0; m < RT; ++m)
#pragma unroll
    for (int i = 0; i < KD; ++i) q[m][i] = *reinterpret_cast<const uint4*>(&sq[quad + 8 * m][i * 32 + j * 8]);
  float o[VT][2 * RT];
#pragma unroll
  for (int t = 0; t < VT; ++t)
#pragma unroll
    for (int e = 0; e < 2 * RT; ++e) o[t][e] = 0.f;
  float mx[RT], l[RT];
#pragma unroll
  for (int m = 0; m < RT; ++m) {
    mx[m] = -INFINITY;
    l[m] = 0.f;
  }
  const float sc = p.scale * 1.4426950408889634f;
  for (int n = 0; n < mine; ++n) {
    prefetch(n + p.stages - 1);
    if (p.stages == 2) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else if (p.stages == 3) asm volatile("cp.async.wait_group 2;" ::: "memory");
    else asm volatile("cp.async.wait_group 3;" ::: "memory");
    __syncwarp();
    uint8_t* st = ring + (n % p.stages) * stage_bytes;
    const int blk = blk0 + warp + n * WD_WARPS, key0 = first_key(blk), end = end_key(blk);
    if (blk == blocks - 1) {  // the new key and value take their place
      const int k = pos - key0;
      for (int i = lane; i < KD * 4; i += 32)
        *reinterpret_cast<uint4*>(st + (((k >> 3) * KD + (i >> 2)) * 32 + (k & 7) * 4 + (i & 3)) * 16) =
            *reinterpret_cast<const uint4*>(&sq[HEADS][i * 8]);
      for (int i = lane; i < p.vdim / 8; i += 32)
        *reinterpret_cast<uint4*>(st + KEYS * KD * 64 + (k * vld + i * 8) * 2) = *reinterpret_cast<const uint4*>(v_new + i * 8);
      __syncwarp();
    }
    float s[KT][2 * RT];
#pragma unroll
    for (int t = 0; t < KT; ++t) {
#pragma unroll
      for (int e = 0; e < 2 * RT; ++e) s[t][e] = 0.f;
#pragma unroll
      for (int i = 0; i < KD; ++i) {
        const uint4 k = *reinterpret_cast<const uint4*>(st + ((t * KD + i) * 32 + lane) * 16);
        const uint4 &lo = q[0][i], &hi = q[RT - 1][i];
        wd_mma(s[t], make_uint2(lo.x, lo.y), make_uint2(hi.x, hi.y), k.x, k.y);
        wd_mma(s[t], make_uint2(lo.z, lo.w), make_uint2(hi.z, hi.w), k.z, k.w);
      }
#pragma unroll
      for (int e = 0; e < 2 * RT; ++e)
        s[t][e] = key0 + t * 8 + 2 * j + (e & 1) < end ? s[t][e] * sc : -INFINITY;
    }
    float alpha[RT];
    uint2 ph[KT / 2][RT], pl[KT / 2][RT];  // weights as operands of the second product, and their rounding errors
#pragma unroll
    for (int m = 0; m < RT; ++m) {
      float v = -INFINITY;
#pragma unroll
      for (int t = 0; t < KT; ++t) v = fmaxf(v, fmaxf(s[t][2 * m], s[t][2 * m + 1]));
      v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
      v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
      const float m_new = fmaxf(mx[m], v);  // finite: the first key of a block is always visible
      alpha[m] = exp2f(mx[m] - m_new);
      mx[m] = m_new;
      float sum = 0.f;
#pragma unroll
      for (int t = 0; t < KT; ++t) {
        const float x = exp2f(s[t][2 * m] - m_new), y = exp2f(s[t][2 * m + 1] - m_new);
        sum += x + y;
        const uint32_t hi = dd_pack(x, y), lo = dd_pack(x - dd_lo(hi), y - dd_hi(hi));
        uint2 &h = ph[t / 2][m], &r = pl[t / 2][m];
        (t % 2 ? h.y : h.x) = hi;
        (t % 2 ? r.y : r.x) = lo;
      }
      l[m] = l[m] * alpha[m] + sum;  // this lane's share of the row sum
    }
    bool moved = false;
#pragma unroll
    for (int m = 0; m < RT; ++m) moved |= alpha[m] != 1.f;
    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
      for (int t = 0; t < VT; ++t)
#pragma unroll
        for (int e = 0; e < 2 * RT; ++e) o[t][e] *= alpha[e >> 1];
    }
    const uint32_t sv = (uint32_t)__cvta_generic_to_shared(st + KEYS * KD * 64);
    const uint32_t vaddr = sv + (((lane & 7) + ((lane >> 3) & 1) * 8) * vld + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int t = 0; t < VT; t += 2) {
      if (t * 8 < p.vdim) {
#pragma unroll
        for (int k = 0; k < KT / 2; ++k) {
          uint32_t v0, v1, v2, v3;  // 16 keys of value tiles t (v0, v1) and t + 1 (v2, v3)
          asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                       : "=r"(v0), "=r"(v1), "=r"(v2), "=r"(v3)
                       : "r"(vaddr + k * 32 * vld + t * 16));
          wd_mma(o[t], ph[k][0], ph[k][RT - 1], v0, v1);
          wd_mma(o[t + 1], ph[k][0], ph[k][RT - 1], v2, v3);
          wd_mma(o[t], pl[k][0], pl[k][RT - 1], v0, v1);
          wd_mma(o[t + 1], pl[k][0], pl[k][RT - 1], v2, v3);
        }
      }
    }
    __syncwarp();  // every lane has read the stage before it is refilled
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int m = 0; m < RT; ++m) {
    l[m] += __shfl_xor_sync(0xffffffffu, l[m], 1);
    l[m] += __shfl_xor_sync(0xffffffffu, l[m], 2);
    if (j == 0) {
      sm[warp][quad + 8 * m] = mx[m];
      sl[warp][quad + 8 * m] = l[m];
    }
  }
  __syncthreads();  // all rings are idle: their memory holds the warps' outputs from here on
  float* so = reinterpret_cast<float*>(smem);  // [WD_WARPS][HEADS][vdim]
#pragma unroll
  for (int t = 0; t < VT; ++t) {
    if (t * 8 < p.vdim) {
#pragma unroll
      for (int m = 0; m < RT; ++m)
        *reinterpret_cast<float2*>(so + ((long long)warp * HEADS + quad + 8 * m) * p.vdim + t * 8 + 2 * j) =
            make_float2(o[t][2 * m], o[t][2 * m + 1]);
    }
  }
  // ---- merge of the warps; the slice's result goes to `part`, or stays here when there is one slice ------------------------
  __shared__ float fm[HEADS], fl[HEADS];
  const long long unit = (long long)b * gridDim.y + blockIdx.y;
  const int pw = p.vdim + 2;
  const float sink = p.sink * 1.4426950408889634f;
  float* mypart = p.part + (unit * splits + split) * HEADS * pw;
  if (threadIdx.x < HEADS) {
    const int r = threadIdx.x;
    float m = splits > 1 ? -INFINITY : sink;
    for (int w = 0; w < WD_WARPS; ++w) m = fmaxf(m, sm[w][r]);
    float ll = splits > 1 || sink == -INFINITY ? 0.f : exp2f(sink - m);
    for (int w = 0; w < WD_WARPS; ++w) ll += sm[w][r] == -INFINITY ? 0.f : sl[w][r] * exp2f(sm[w][r] - m);
    fm[r] = m;
    fl[r] = ll;
    if (splits > 1) {
      __stcg(mypart + r * pw, m);
      __stcg(mypart + r * pw + 1, ll);
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * p.vdim; i += blockDim.x) {
    const int r = i / p.vdim, c = i - r * p.vdim;
    float acc = 0.f;
#pragma unroll
    for (int w = 0; w < WD_WARPS; ++w)
      acc += sm[w][r] == -INFINITY ? 0.f : so[((long long)w * HEADS + r) * p.vdim + c] * exp2f(sm[w][r] - fm[r]);
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
    const float* parts = p.part + unit * splits * HEADS * pw;
    for (int i = threadIdx.x; i < splits * HEADS; i += blockDim.x) {
      wt[i] = __ldcg(parts + (long long)i * pw);
      wl[i] = __ldcg(parts + (long long)i * pw + 1);
    }
    __syncthreads();
    if (threadIdx.x < HEADS) {
      float m = sink;
      for (int k = 0; k < splits; ++k) m = fmaxf(m, wt[k * HEADS + threadIdx.x]);
      float ll = sink == -INFINITY ? 0.f : exp2f(sink - m);
      for (int k = 0; k < splits; ++k) {
        float& w = wt[k * HEADS + threadIdx.x];
        w = w == -INFINITY ? 0.f : exp2f(w - m);
        ll += w * wl[k * HEADS + threadIdx.x];
      }
      fl[threadIdx.x] = ll;
    }
    if (threadIdx.x == 0) p.counters[unit] = 0;
  }
  __syncthreads();
  const float* parts = p.part + unit * splits * HEADS * pw;
  const __nv_bfloat16* gate = row + (long long)(p.H + p.G) * p.dim + (long long)p.G * p.vdim + (long long)h0 * p.vdim;
  for (int i = threadIdx.x; i < nh * p.vdim; i += blockDim.x) {
    const int r = i / p.vdim, c = i - r * p.vdim;
    float acc = 0.f;
    if (splits > 1) {
      const float* src = parts + (long long)r * pw + 2 + c;
#pragma unroll 8
      for (int k = 0; k < splits; ++k) acc += wt[k * HEADS + r] * __ldcg(src + (long long)k * HEADS * pw);
    } else {
      acc = so[(long long)r * p.vdim + c];
    }
    acc /= fl[r];
    if (p.gated) acc *= gate_factor(__bfloat162float(gate[i]));
    p.out[(long long)b * p.ldo + (long long)h0 * p.vdim + i] = __float2bfloat16_rn(acc);
  }
}

constexpr int WD_RING_LIMIT = 104 * 1024;  // two CTAs per SM

template <int KD, int VT, int RT> int wd_launch_rows(WindowDecodeParams p, int B, int splits, cudaStream_t s) {
  const int stage = wd_stage_bytes(wd_keys(KD, VT), KD, p.vdim) * WD_WARPS;
  p.stages = 4 * stage <= WD_RING_LIMIT ? 4 : (3 * stage <= WD_RING_LIMIT ? 3 : 2);
  int bytes = p.stages * stage;
  const int merge = WD_WARPS * 8 * RT * p.vdim * 4;
  if (bytes < merge) bytes = merge;
  static int configured = 0;
  if (configured < bytes) {
    const cudaError_t e =
        cudaFuncSetAttribute(window_attn_decode_kernel<KD, VT, RT>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return (int)e;
    configured = bytes;
  }
  const int hchunks = (p.H / p.G + 8 * RT - 1) / (8 * RT);
  const cudaError_t e = xl_launch_overlapped(window_attn_decode_kernel<KD, VT, RT>, dim3(splits, p.G * hchunks, B),
                                             dim3(WD_WARPS * 32), (size_t)bytes, s, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

template <int KD, int VT> int wd_launch(const WindowDecodeParams& p, int B, int splits, cudaStream_t s) {
  return p.H / p.G <= 8 ? wd_launch_rows<KD, VT, 1>(p, B, splits, s) : wd_launch_rows<KD, VT, 2>(p, B, splits, s);
}

}  // namespace

// proj: (B*T_len, ld) as described above; wq, wk (dim) fp32; qn (B, G, T_len, H/G, dim). dim <= 512. Rows past count[b] are
// left out.
XL_API int xl_qk_norm_append(const void* proj, long long ld, const float* wq, const float* wk, void* qn, void* kc, void* vc,
                             const int* pos, const int* count, int B, int T_len, int H, int G, int dim, int vdim, int Smax,
                             float eps, int dtype, cudaStream_t s) {
  if (B < 1 || B > 65535 || T_len < 1 || G < 1 || H < 1 || H % G || dim < 1 || dim > WA_MAX_DIM || vdim < 1 || Smax < 1 ||
      ld < (long long)(H + G) * dim + (long long)G * vdim || !wq || !wk)
    return -1;
  XL_DISPATCH_DTYPE(dtype, T, {
    constexpr int V = 16 / sizeof(T);
    if (dim % V == 0 && vdim % V == 0 && ld % V == 0 && (((uintptr_t)proj | (uintptr_t)qn | (uintptr_t)kc | (uintptr_t)vc) & 15) == 0)
      return launch_append<T, V>(proj, ld, wq, wk, qn, kc, vc, pos, count, B, T_len, H, G, dim, vdim, Smax, eps, s);
    return launch_append<T, 1>(proj, ld, wq, wk, qn, kc, vc, pos, count, B, T_len, H, G, dim, vdim, Smax, eps, s);
  });
  return (int)cudaGetLastError();
}

// qn as above; gate: first gate column of the projections (row stride ldg), or null; out: (B*T_len, ldo). dim <= 512, vdim <= 512.
// Rows past count[b] of a sequence are left as they are.
XL_API int xl_window_attn_general(const void* qn, const void* kc, const void* vc, const void* gate, long long ldg, void* out,
                                  long long ldo, const int* pos, const int* count, int B, int T_len, int H, int G, int dim,
                                  int vdim, int Smax, int window, int keep_first, float scale, float sink, int dtype,
                                  cudaStream_t s) {
  if (B < 1 || B > 65535 || H < 1 || H > 65535 || T_len < 1 || G < 1 || H % G || dim < 1 || dim > WA_MAX_DIM || vdim < 1 ||
      vdim > 512 || Smax < 1 || window < 0 || keep_first < 0)
    return -1;
  const dim3 grid((T_len + WG_WARPS - 1) / WG_WARPS, H, B);
#define XL_WG(VPL)                                                                                                            \
  window_attn_general_kernel<T, VPL><<<grid, WG_WARPS * 32, 0, s>>>((const T*)qn, (const T*)kc, (const T*)vc, (const T*)gate,    \
                                                                    ldg, (T*)out, ldo, pos, count, T_len, H, G, dim, vdim, Smax, \
                                                                    window, keep_first, scale, sink)
  XL_DISPATCH_DTYPE(dtype, T, {
    if (vdim <= 128) XL_WG(4);
    else XL_WG(16);
  });
#undef XL_WG
  return (int)cudaGetLastError();
}

// One token per sequence (rows of proj = sequences), bf16. dim, vdim multiples of 8, dim <= 128, vdim <= 256, ld a multiple of
// 8. The kernel normalises q and k and appends; proj is not modified. gated: proj rows end in gate columns. part: B * G *
// ceil(H/G/16) * splits * 16 * (vdim + 2) floats; counters: B * G * ceil(H/G/16) zero-initialised words (left zeroed). Sequences
// with count 0 are skipped. The kernel may read the caches before its predecessor on the stream has ended.
XL_API int xl_window_attn_decode(const void* proj, long long ld, const float* wq, const float* wk, void* kc, void* vc, void* out,
                                 long long ldo, const int* pos, const int* count, int B, int H, int G, int dim, int vdim, int Smax,
                                 int window, int keep_first, int gated, float scale, float sink, float eps, int splits,
                                 float* part, unsigned int* counters, cudaStream_t s) {
  if (B < 1 || B > 65535 || G < 1 || H < 1 || H % G || H > 4096 || dim < 8 || dim > 128 || dim % 8 || vdim < 8 || vdim > 256 ||
      vdim % 8 || Smax < 1 || window < 0 || keep_first < 0 || splits < 1 || splits > WD_MAX_SPLITS || (ld % 8) || !wq || !wk ||
      ld < (long long)(H + G) * dim + (long long)G * vdim + (gated ? (long long)H * vdim : 0) || ldo < (long long)H * vdim)
    return -1;
  if (((uintptr_t)proj & 15) || ((uintptr_t)kc & 15) || ((uintptr_t)vc & 15)) return -1;
  if (splits > 1 && (!part || !counters)) return -1;
  WindowDecodeParams p = {};
  p.proj = (const __nv_bfloat16*)proj; p.ld = ld; p.wq = wq; p.wk = wk;
  p.kc = (__nv_bfloat16*)kc; p.vc = (__nv_bfloat16*)vc; p.out = (__nv_bfloat16*)out; p.ldo = ldo;
  p.pos = pos; p.count = count; p.H = H; p.G = G; p.dim = dim; p.vdim = vdim; p.Smax = Smax; p.window = window;
  p.keep_first = keep_first; p.gated = gated; p.scale = scale; p.sink = sink; p.eps = eps; p.part = part; p.counters = counters;
#define XL_WD(KD)                                             \
  if (vdim <= 64) return wd_launch<KD, 8>(p, B, splits, s);   \
  if (vdim <= 128) return wd_launch<KD, 16>(p, B, splits, s); \
  return wd_launch<KD, 32>(p, B, splits, s);
  if (dim <= 32) { XL_WD(1) }
  if (dim <= 64) { XL_WD(2) }
  XL_WD(4)
#undef XL_WD
}
