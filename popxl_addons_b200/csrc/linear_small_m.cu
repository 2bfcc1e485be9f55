// Linear layers of the decoding path, bf16 weights, M <= 16 rows: C[M, N] = a[M, K] * w[N, K]^T, the weights streamed once.
// What follows the product in a layer happens in the epilogue, on the fp32 sums:
//   store      C as bf16 or fp32
//   residual   x += mult * C (+ table[token]) on the fp32 residual stream; for the next layer h = DyT(x), or the first half of
//              an RMS norm: h = x * w and the sums of squares of x over blocks of 64 columns (one column tile each)
//   swiglu     weight rows [gate | up]: y = silu(gate) * up
//   split_glu  weight rows [plain | gate | up]: plain results stored, a clamped gated unit of the others beside them
//   min_gru    weight rows [z | u | g], one row per sequence: one step of the recurrence on the fp32 state
//
// store and split_glu may take rows of such a half-done norm: their results are multiplied by 1 / sqrt(mean(x^2) + eps), summed
// up from the blocks' sums of squares while the weights arrive.
//
// The product is bandwidth-bound (at most 16 multiply-adds per weight), so it uses `mma.sync.m16n8k16` with operands from
// registers: each lane copies two 16-byte pieces of a weight row (four lanes: 64 contiguous bytes each time) through a per-warp
// cp.async ring and feeds them to four MMAs; the activations it needs for them are loaded one chunk ahead into registers. (Any assignment of k indices to the k slots of an MMA is valid as long as both operands agree.)
//
// Work = (column tiles) x (K chunks of 64), tile-major, cut into equal contiguous ranges, one per CTA, so the grid fits the
// machine and not the problem. A tile shared by several CTAs is finished by the one that arrives last: every CTA leaves its
// partial sums in a slot of its own and the finisher adds the slots in CTA order, so results do not depend on timing.
// No CTA waits for another. Consecutive kernels overlap: a launch requests its first weights while its predecessor drains. An epilogue that combines several weight rows per output channel (swiglu, min_gru) takes them
// into one tile: a tile is PARTS groups of CH channels, group p starting at weight row p * N / PARTS.
#include "common.cuh"

#include <math.h>

namespace {

constexpr int SM_WARPS = 4;
constexpr int SM_KC = 64;       // k values per chunk (16 per lane)
constexpr int SM_STAGES = 3;
constexpr int SM_CTAS_PER_SM = 2;

enum SmMode : int { SM_STORE = 0, SM_RESIDUAL = 1, SM_SWIGLU = 2, SM_MINGRU = 3, SM_SPLIT_GLU = 4 };

// split_glu has two kinds of tiles: first those of the plain rows (one part of 64 channels), then those of the gated unit.
template <int MODE> struct SmTile {
  static constexpr int PARTS = MODE == SM_SWIGLU || MODE == SM_SPLIT_GLU ? 2 : (MODE == SM_MINGRU ? 3 : 1);
  static constexpr int CH = PARTS == 2 ? 32 : (MODE == SM_MINGRU ? 16 : 64);  // channels per tile
  static constexpr int COLS = PARTS * CH;
  static constexpr int NT = COLS / 8;
  static constexpr int STAGE = NT * 2 * 32;  // uint4: two pieces of NT weight rows per lane
  static constexpr int RING_BYTES = SM_WARPS * SM_STAGES * STAGE * 16;
};

struct SmParams {
  const __nv_bfloat16* a;
  long long lda;
  const __nv_bfloat16* w;  // (N, K), contiguous
  int M, N, K;
  // store / swiglu / min_gru
  void* y;
  long long ldy;
  int y_f32;
  // residual
  float* x;
  float mult;
  const int* tokens;
  const __nv_bfloat16* table;
  int vocab;
  const float *alpha, *nw, *nb;  // DyT; alpha null: h = x * nw and the sums of squares
  __nv_bfloat16* h;
  float* sumsq_out;  // (M, column tiles)
  // store / split_glu: sums of squares of the rows of a half-done norm, (M, sumsq_parts), or null
  const float* sumsq;
  int sumsq_parts;
  float eps;
  // split_glu: y holds the plain results, z the unit's
  int cols;
  __nv_bfloat16* z;
  long long ldz;
  float limit, slope, shift;
  // min_gru
  const float *bz, *bu;
  float* state;
  const int *pos, *count;
  // split-K scratch
  float* slots;            // [grid][2][16 * COLS]
  unsigned int* counters;  // one per tile, zero between launches
};

__device__ __forceinline__ void cp_async16(uint4* dst, const void* src, bool on) {
  const int bytes = on ? 16 : 0;  // 0: the destination is zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src),
               "r"(bytes)
               : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float sigmoid_f(float v) { return 1.f / (1.f + expf(-v)); }
__device__ __forceinline__ float silu_f(float v) { return v / (1.f + expf(-v)); }

// Four channels c .. c + 3 of row r (those below `channels`). All loads come before the first store: their latencies overlap.
// Returns the sum of squares of what it wrote to the residual stream.
template <int MODE>
__device__ __forceinline__ float sm_epilogue(const SmParams& p, int r, int c, const float (&v)[SmTile<MODE>::PARTS][4], int channels,
                                             bool unit) {
  constexpr int LAST = SmTile<MODE>::PARTS - 1;
  const int n = min(4, channels - c);
  float sq = 0.f;
  const long long at = (long long)r * channels + c, yat = (long long)r * p.ldy + c;
  if (MODE == SM_SPLIT_GLU && unit) {
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (e < n)
        p.z[(long long)r * p.ldz + c + e] =
            __float2bfloat16_rn(xl_clamped_glu_value(v[0][e], v[LAST][e], p.limit, p.slope, p.shift));
  } else if (MODE == SM_STORE || MODE == SM_SPLIT_GLU) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (e < n) {
        if (p.y_f32) ((float*)p.y)[yat + e] = v[0][e];
        else ((__nv_bfloat16*)p.y)[yat + e] = __float2bfloat16_rn(v[0][e]);
      }
    }
  } else if (MODE == SM_RESIDUAL) {
    float x[4], add[4], nw[4], nb[4];
    const __nv_bfloat16* row = p.table ? p.table + (long long)min(max(p.tokens[r], 0), p.vocab - 1) * channels + c : nullptr;
    const float alpha = p.alpha ? *p.alpha : 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = e < n ? e : 0;
      x[e] = p.x[at + k];
      add[e] = row ? __bfloat162float(row[k]) : 0.f;
      nw[e] = p.nw ? p.nw[c + k] : 0.f;
      nb[e] = p.alpha ? p.nb[c + k] : 0.f;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (e < n) {
        const float s = x[e] + p.mult * v[0][e] + add[e];
        p.x[at + e] = s;
        sq += s * s;
        if (p.alpha) p.h[at + e] = __float2bfloat16_rn(tanhf(alpha * s) * nw[e] + nb[e]);
        else if (p.nw) p.h[at + e] = __float2bfloat16_rn(s * nw[e]);
      }
    }
  } else if (MODE == SM_SWIGLU) {
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (e < n) ((__nv_bfloat16*)p.y)[yat + e] = __float2bfloat16_rn(silu_f(v[0][e]) * v[LAST][e]);
  } else {
    float old[4], bz[4], bu[4];
    const bool fresh = p.pos[r] <= 0, real = p.count[r] > 0;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = e < n ? e : 0;
      old[e] = fresh ? 0.f : p.state[at + k];
      bz[e] = p.bz[c + k];
      bu[e] = p.bu[c + k];
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (e < n) {
        const float z = sigmoid_f(v[0][e] + bz[e]), u = v[1 % SmTile<MODE>::PARTS][e] + bu[e];
        float s = old[e];
        if (real) {
          s = (1.f - z) * s + z * (u >= 0.f ? u + 0.5f : sigmoid_f(u));
          p.state[at + e] = s;
        }
        ((__nv_bfloat16*)p.y)[yat + e] = __float2bfloat16_rn(s * silu_f(v[LAST][e]));
      }
    }
  }
  return sq;
}

// Contiguous ranges of items: the first `rem` CTAs take per + 1 items, the others per.
struct SmRanges {
  int per, rem;
  __device__ __forceinline__ int begin(int cta) const { return cta * per + min(cta, rem); }
  __device__ __forceinline__ int owner(int item) const {
    const int head = rem * (per + 1);
    return item < head ? item / (per + 1) : rem + (item - head) / per;
  }
};

template <int MODE>
__global__ void __launch_bounds__(SM_WARPS * 32, SM_CTAS_PER_SM) linear_small_m_kernel(const SmParams p) {
  using L = SmTile<MODE>;
  constexpr int NT = L::NT, COLS = L::COLS, CH = L::CH, PARTS = L::PARTS;
  extern __shared__ uint4 ring_all[];
  __shared__ float red[SM_WARPS][16][COLS + 1];
  __shared__ unsigned int finish;
  __shared__ float row_scale[16];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int quad = lane >> 2, j = lane & 3;
  const int chunks = (p.K + SM_KC - 1) / SM_KC;
  // tiles [0, plain) have one part of COLS channels (split_glu only), the others PARTS parts of CH
  const int plain = MODE == SM_SPLIT_GLU ? (p.cols + COLS - 1) / COLS : 0;
  const int channels = MODE == SM_SPLIT_GLU ? (p.N - p.cols) / PARTS : p.N / PARTS;
  const int n_tiles = plain + (channels + CH - 1) / CH;
  const int total = n_tiles * chunks;
  const SmRanges ranges{total / (int)gridDim.x, total % (int)gridDim.x};
  int item = ranges.begin(blockIdx.x);
  const int item_end = ranges.begin(blockIdx.x + 1);
  const int first_tile = item / chunks;
  uint4* ring = ring_all + warp * (SM_STAGES * L::STAGE);

  // The chunks of this warp over the whole range, tile after tile: (tile, chunk) of the next one to request and of the next to
  // multiply advance by the same rule.
  struct Cursor { int item, c1, ch, tile; };  // first item of the current tile segment, its end chunk, current chunk
  auto segment = [&](Cursor& c) {  // enter the segment that starts at c.item (or stop at the end of the range)
    while (c.item < item_end) {
      c.tile = c.item / chunks;
      const int c0 = c.item - c.tile * chunks;
      c.c1 = min(chunks, c0 + (item_end - c.item));
      c.ch = c0 + warp;
      if (c.ch < c.c1) return;
      c.item += c.c1 - c0;
    }
  };
  auto advance = [&](Cursor& c) {
    c.ch += SM_WARPS;
    if (c.ch >= c.c1) {
      c.item = c.tile * chunks + c.c1;
      segment(c);
    }
  };
  auto request = [&](const Cursor& c, int buf) {
    if (c.item < item_end) {
      const int k0 = c.ch * SM_KC + j * 8;
      uint4* dst = ring + buf * L::STAGE + lane;
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        const int col = t * 8 + quad;
        bool row_on;
        long long w_row;
        if (MODE == SM_SPLIT_GLU && c.tile < plain) {
          w_row = c.tile * COLS + col;
          row_on = w_row < p.cols;
        } else {
          const int n = (c.tile - plain) * CH + col % CH;
          row_on = n < channels;
          w_row = (MODE == SM_SPLIT_GLU ? p.cols : 0) + (long long)(col / CH) * channels + n;
        }
        const __nv_bfloat16* src = p.w + (row_on ? w_row : 0) * p.K;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const bool on = row_on && k0 + e * 32 < p.K;
          cp_async16(dst + (t * 2 + e) * 32, src + (on ? k0 + e * 32 : 0), on);
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");  // possibly empty: one group per chunk slot
  };
  auto load_a = [&](const Cursor& c, uint4 (&lo)[2], uint4 (&hi)[2]) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int k = c.ch * SM_KC + j * 8 + e * 32;
      const bool on = c.item < item_end && k < p.K;
      lo[e] = on && quad < p.M ? *reinterpret_cast<const uint4*>(p.a + (long long)quad * p.lda + k) : make_uint4(0, 0, 0, 0);
      hi[e] = on && quad + 8 < p.M ? *reinterpret_cast<const uint4*>(p.a + (long long)(quad + 8) * p.lda + k) : make_uint4(0, 0, 0, 0);
    }
  };
  Cursor ahead{item, 0, 0, 0};
  segment(ahead);
  Cursor cur = ahead;
#pragma unroll
  for (int n = 0; n < SM_STAGES - 1; ++n) {
    request(ahead, n);
    if (ahead.item < item_end) advance(ahead);
  }
  xl_grid_dependency_wait();  // the first weights are on their way; everything else may come from the previous kernel
  xl_grid_launch_dependents();
  uint4 a_lo[2], a_hi[2];
  load_a(cur, a_lo, a_hi);
  if ((MODE == SM_STORE || MODE == SM_SPLIT_GLU) && p.sumsq) {  // read after the barriers of the first tile
    for (int r = warp; r < p.M; r += SM_WARPS) {
      float sq = 0.f;
      for (int i = lane; i < p.sumsq_parts; i += 32) sq += p.sumsq[(long long)r * p.sumsq_parts + i];
      sq = xl_warp_sum(sq);
      if (lane == 0) row_scale[r] = 1.f / sqrtf(sq / p.K + p.eps);
    }
  }
  int buf = 0;
  while (item < item_end) {
    const int tile = item / chunks;
    const int c0 = item - tile * chunks;
    const int c1 = min(chunks, c0 + (item_end - item));
    float acc[NT][4];
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[t][e] = 0.f;
    for (int ch = c0 + warp; ch < c1; ch += SM_WARPS) {
      request(ahead, (buf + SM_STAGES - 1) % SM_STAGES);
      if (ahead.item < item_end) advance(ahead);
      uint4 lo[2] = {a_lo[0], a_lo[1]}, hi[2] = {a_hi[0], a_hi[1]};
      advance(cur);
      load_a(cur, a_lo, a_hi);
      asm volatile("cp.async.wait_group %0;" ::"n"(SM_STAGES - 1) : "memory");
      const uint4* src = ring + buf * L::STAGE + lane;  // every lane reads back the pieces it copied itself
      buf = (buf + 1) % SM_STAGES;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint4 w[NT];
#pragma unroll
        for (int t = 0; t < NT; ++t) w[t] = src[(t * 2 + e) * 32];
#pragma unroll
        for (int t = 0; t < NT; ++t) mma_bf16(acc[t], lo[e].x, hi[e].x, lo[e].y, hi[e].y, w[t].x, w[t].y);
#pragma unroll
        for (int t = 0; t < NT; ++t) mma_bf16(acc[t], lo[e].z, hi[e].z, lo[e].w, hi[e].w, w[t].z, w[t].w);
      }
    }
    __syncthreads();  // readers of the previous tile are done with `red`
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      red[warp][quad][t * 8 + 2 * j] = acc[t][0];
      red[warp][quad][t * 8 + 2 * j + 1] = acc[t][1];
      red[warp][quad + 8][t * 8 + 2 * j] = acc[t][2];
      red[warp][quad + 8][t * 8 + 2 * j + 1] = acc[t][3];
    }
    __syncthreads();
    const bool whole = c1 - c0 == chunks;
    bool finishing = whole;
    if (!whole) {
      float* slot = p.slots + ((long long)blockIdx.x * 2 + (tile == first_tile ? 0 : 1)) * (16 * COLS);
      for (int i = threadIdx.x; i < p.M * COLS; i += blockDim.x) {
        const int r = i / COLS, col = i % COLS;
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < SM_WARPS; ++w) s += red[w][r][col];
        __stcg(slot + i, s);
      }
      __threadfence();
      __syncthreads();
      if (threadIdx.x == 0)
        finish = atomicAdd(p.counters + tile, (unsigned int)(c1 - c0)) + (unsigned int)(c1 - c0) == (unsigned int)chunks;
      __syncthreads();
      finishing = finish != 0;
      if (finishing) __threadfence();
    }
    if (finishing) {
      // CTAs that share the tile, in order. All but the first begin inside it: it is their first tile (slot 0). It is the
      // last tile of the first one, and its first only if that one begins exactly with it.
      int cta0 = blockIdx.x, cta1 = blockIdx.x, slot0 = 0;
      if (!whole) {
        cta0 = ranges.owner(tile * chunks);
        cta1 = ranges.owner(tile * chunks + chunks - 1);
        slot0 = ranges.begin(cta0) < tile * chunks ? 1 : 0;
      }
      const bool unit = tile >= plain;  // one part of COLS channels, or PARTS parts of CH
      const int ch = MODE == SM_SPLIT_GLU && !unit ? COLS : CH, parts = MODE == SM_SPLIT_GLU && !unit ? 1 : PARTS;
      const int end = MODE == SM_SPLIT_GLU && !unit ? p.cols : channels, per_row = ch / 4;
      for (int i = threadIdx.x; i < p.M * per_row; i += blockDim.x) {
        const int r = i / per_row, cc = (i % per_row) * 4, c = (unit ? tile - plain : tile) * ch + cc;
        float sq = 0.f;
        if (c < end) {
          float v[PARTS][4];
#pragma unroll
          for (int q = 0; q < PARTS; ++q) {
            const int col = q * CH + cc;
            if (MODE == SM_SPLIT_GLU && q >= parts) {
#pragma unroll
              for (int e = 0; e < 4; ++e) v[q][e] = 0.f;
            } else if (whole) {
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                v[q][e] = 0.f;
#pragma unroll
                for (int w = 0; w < SM_WARPS; ++w) v[q][e] += red[w][r][col + e];
              }
            } else {
              const float* base = p.slots + r * COLS + col;
              float4 t = __ldcg(reinterpret_cast<const float4*>(base + ((long long)cta0 * 2 + slot0) * (16 * COLS)));
#pragma unroll 8
              for (int k = cta0 + 1; k <= cta1; ++k) {
                const float4 o = __ldcg(reinterpret_cast<const float4*>(base + (long long)k * 2 * (16 * COLS)));
                t.x += o.x; t.y += o.y; t.z += o.z; t.w += o.w;
              }
              v[q][0] = t.x; v[q][1] = t.y; v[q][2] = t.z; v[q][3] = t.w;
            }
            if ((MODE == SM_STORE || MODE == SM_SPLIT_GLU) && p.sumsq) {
#pragma unroll
              for (int e = 0; e < 4; ++e) v[q][e] *= row_scale[r];
            }
          }
          sq = sm_epilogue<MODE>(p, r, c, v, end, unit);
        }
        if (MODE == SM_RESIDUAL && p.sumsq_out) {
          // the 16 lanes of a half-warp hold one row; either all or none of them are here
          const unsigned int half = 0xffffu << (lane & 16);
#pragma unroll
          for (int o = 8; o > 0; o >>= 1) sq += __shfl_xor_sync(half, sq, o);
          if ((lane & 15) == 0) p.sumsq_out[(long long)r * n_tiles + tile] = sq;
        }
      }
      if (!whole && threadIdx.x == 0) p.counters[tile] = 0;
    }
    item += c1 - c0;
  }
}

template <int MODE> int sm_launch(const SmParams& p, int sms, int max_tiles, cudaStream_t s) {
  using L = SmTile<MODE>;
  const int paired = MODE == SM_SPLIT_GLU ? p.N - p.cols : p.N;
  if (paired % L::PARTS) return -1;
  const int plain = MODE == SM_SPLIT_GLU ? (p.cols + L::COLS - 1) / L::COLS : 0;
  const int channels = paired / L::PARTS, chunks = (p.K + SM_KC - 1) / SM_KC, n_tiles = plain + (channels + L::CH - 1) / L::CH;
  if (n_tiles > max_tiles) return -1;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e =
        cudaFuncSetAttribute(linear_small_m_kernel<MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::RING_BYTES);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  long long grid = (long long)SM_CTAS_PER_SM * sms;
  const long long total = (long long)n_tiles * chunks;
  if (total > (1 << 30)) return -1;
  if (grid > total) grid = total;
  const cudaError_t e = xl_launch_overlapped(linear_small_m_kernel<MODE>, dim3((unsigned)grid), dim3(SM_WARPS * 32),
                                             L::RING_BYTES, s, p);
  return e != cudaSuccess ? (int)e : (int)cudaGetLastError();
}

int sm_check(const void* a, long long lda, const void* w, int M, int N, int K, const float* slots, const unsigned int* counters) {
  if (M < 1 || M > 16 || N < 1 || K < 8 || (K % 8) || (lda % 8) || lda < K) return -1;
  if (((uintptr_t)a & 15) || ((uintptr_t)w & 15) || !slots || !counters) return -1;
  return 0;
}

}  // namespace

// Floats of `slots` for a device with `sms` SMs; `counters` needs `max_tiles` zero-initialised words (left zeroed).
XL_API int xl_linear_small_m_slots(int sms) { return SM_CTAS_PER_SM * sms * 2 * 16 * 64; }

// All: a (M, K) bf16 with row stride lda (a multiple of 8), w (N, K) bf16 contiguous, M <= 16, K a multiple of 8; returns -1
// for arguments the kernel does not take. y (M, N) with row stride ldy, bf16 or fp32. sumsq (M, sumsq_parts), or null: the rows
// of y are multiplied by 1 / sqrt(sum of the row's sumsq / K + eps).
XL_API int xl_linear_small_m(const void* a, long long lda, const void* w, void* y, long long ldy, int y_f32, const float* sumsq,
                             int sumsq_parts, float eps, int M, int N, int K, float* slots, unsigned int* counters, int max_tiles,
                             int sms, cudaStream_t s) {
  if (sm_check(a, lda, w, M, N, K, slots, counters) || !y || (sumsq && sumsq_parts < 1)) return -1;
  SmParams p = {};
  p.a = (const __nv_bfloat16*)a; p.lda = lda; p.w = (const __nv_bfloat16*)w; p.M = M; p.N = N; p.K = K;
  p.y = y; p.ldy = ldy; p.y_f32 = y_f32; p.sumsq = sumsq; p.sumsq_parts = sumsq_parts; p.eps = eps;
  p.slots = slots; p.counters = counters;
  return sm_launch<SM_STORE>(p, sms, max_tiles, s);
}

// w rows [cols plain | F gate | F up], N = cols + 2F: y (M, cols) with row stride ldy and z (M, F) with row stride ldz, bf16;
// sumsq as in xl_linear_small_m.
XL_API int xl_linear_small_m_split_glu(const void* a, long long lda, const void* w, void* y, long long ldy, int cols, void* z,
                                       long long ldz, float limit, float slope, float shift, const float* sumsq, int sumsq_parts,
                                       float eps, int M, int N, int K, float* slots, unsigned int* counters, int max_tiles,
                                       int sms, cudaStream_t s) {
  if (sm_check(a, lda, w, M, N, K, slots, counters) || cols < 0 || cols > N || (cols && !y) || (cols < N && !z) ||
      (sumsq && sumsq_parts < 1))
    return -1;
  SmParams p = {};
  p.a = (const __nv_bfloat16*)a; p.lda = lda; p.w = (const __nv_bfloat16*)w; p.M = M; p.N = N; p.K = K;
  p.y = y; p.ldy = ldy; p.cols = cols; p.z = (__nv_bfloat16*)z; p.ldz = ldz; p.limit = limit; p.slope = slope; p.shift = shift;
  p.sumsq = sumsq; p.sumsq_parts = sumsq_parts; p.eps = eps; p.slots = slots; p.counters = counters;
  return sm_launch<SM_SPLIT_GLU>(p, sms, max_tiles, s);
}

// x (M, N) fp32 += mult * a w^T; with nw, h (M, N) bf16 = x * nw and sumsq (M, ceil(N / 64)) = sums of x^2 over 64 columns.
XL_API int xl_linear_small_m_residual_rms(const void* a, long long lda, const void* w, float* x, float mult, const float* nw,
                                          void* h, float* sumsq, int M, int N, int K, float* slots, unsigned int* counters,
                                          int max_tiles, int sms, cudaStream_t s) {
  if (sm_check(a, lda, w, M, N, K, slots, counters) || !x || (nw && (!h || !sumsq))) return -1;
  SmParams p = {};
  p.a = (const __nv_bfloat16*)a; p.lda = lda; p.w = (const __nv_bfloat16*)w; p.M = M; p.N = N; p.K = K;
  p.x = x; p.mult = mult; p.nw = nw; p.h = (__nv_bfloat16*)h; p.sumsq_out = nw ? sumsq : nullptr;
  p.slots = slots; p.counters = counters;
  return sm_launch<SM_RESIDUAL>(p, sms, max_tiles, s);
}

// x (M, N) fp32 += mult * a w^T (+ table[tokens]); with alpha, h (M, N) bf16 = tanh(alpha x) nw + nb.
XL_API int xl_linear_small_m_residual(const void* a, long long lda, const void* w, float* x, float mult, const int* tokens,
                                      const void* table, int vocab, const float* alpha, const float* nw, const float* nb,
                                      void* h, int M, int N, int K, float* slots, unsigned int* counters, int max_tiles, int sms,
                                      cudaStream_t s) {
  if (sm_check(a, lda, w, M, N, K, slots, counters) || !x || (table && (!tokens || vocab < 1)) || (alpha && (!nw || !nb || !h)))
    return -1;
  SmParams p = {};
  p.a = (const __nv_bfloat16*)a; p.lda = lda; p.w = (const __nv_bfloat16*)w; p.M = M; p.N = N; p.K = K;
  p.x = x; p.mult = mult; p.tokens = tokens; p.table = (const __nv_bfloat16*)table; p.vocab = vocab;
  p.alpha = alpha; p.nw = nw; p.nb = nb; p.h = (__nv_bfloat16*)h; p.slots = slots; p.counters = counters;
  return sm_launch<SM_RESIDUAL>(p, sms, max_tiles, s);
}

// w rows [gate | up] (2F, K); y (M, F) bf16 contiguous.
XL_API int xl_linear_small_m_swiglu(const void* a, long long lda, const void* w, void* y, int M, int F, int K, float* slots,
                                    unsigned int* counters, int max_tiles, int sms, cudaStream_t s) {
  if (sm_check(a, lda, w, M, 2 * F, K, slots, counters) || !y) return -1;
  SmParams p = {};
  p.a = (const __nv_bfloat16*)a; p.lda = lda; p.w = (const __nv_bfloat16*)w; p.M = M; p.N = 2 * F; p.K = K;
  p.y = y; p.ldy = F; p.slots = slots; p.counters = counters;
  return sm_launch<SM_SWIGLU>(p, sms, max_tiles, s);
}

// w rows [z | u | g] (3W, K); row r is the next token of sequence r: state (M, W) fp32 advances where count[r] > 0 and starts
// from zero at pos[r] == 0; y (M, W) bf16 contiguous.
XL_API int xl_linear_small_m_min_gru(const void* a, long long lda, const void* w, const float* bz, const float* bu, float* state,
                                     const int* pos, const int* count, void* y, int M, int W, int K, float* slots,
                                     unsigned int* counters, int max_tiles, int sms, cudaStream_t s) {
  if (sm_check(a, lda, w, M, 3 * W, K, slots, counters) || !y || !state || !bz || !bu || !pos || !count) return -1;
  SmParams p = {};
  p.a = (const __nv_bfloat16*)a; p.lda = lda; p.w = (const __nv_bfloat16*)w; p.M = M; p.N = 3 * W; p.K = K;
  p.y = y; p.ldy = W; p.bz = bz; p.bu = bu; p.state = state; p.pos = pos; p.count = count; p.slots = slots; p.counters = counters;
  return sm_launch<SM_MINGRU>(p, sms, max_tiles, s);
}
