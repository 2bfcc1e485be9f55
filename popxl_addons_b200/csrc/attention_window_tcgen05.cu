// Sliding-window attention of a portion of tokens against the key / value cache on the 5th-generation tensor cores (tcgen05),
// bf16. Same mathematics and layouts as attention_window.cu: visible are a window and the first tokens, a sink in the softmax, a
// gate on the output.
//
// The R query heads that read one key / value head are consecutive rows (token-major) of the normalised queries. One CTA owns
// 256 of these rows as two tiles of 128 and walks the keys visible to any of them in blocks of 128 - first those of the kept
// first tokens, then those of the windows; key and value tiles serve both row tiles:
//   warp 0       TMA producer : both query tiles once, key tiles (lane 0) and value tiles (lane 1) through rings
//   warp 1       MMA issuer   : S_m = Q_m K^T into TMEM, then O_m += P_m V, the two tiles taking turns, so that the softmax of one
//                               runs under the products of the other
//   warps 2..5   softmax of tile 0, warps 6..9 of tile 1: one thread per row; running maximum and sum in fp32 start with the
//                               sink, lazy rescaling of O_m in TMEM
// P replaces S in TMEM as two bf16 numbers per weight (value and rounding error), so the weights keep more than 16 bits.
//
// TMEM columns: [0, 128) S_0 / P_0, [128, 256) S_1 / P_1 (the upper half of each holds the rounding errors),
// [256, 256 + VD) O_0, [256 + VD, 256 + 2 VD) O_1. One CTA per SM. Every wait is bounded (see tcgen05.cuh).
#include "attention_window.cuh"
#include "tcgen05.cuh"

namespace {

constexpr int TILE_M = 128;
constexpr int BKV = 128;
constexpr int UMMA_K = 16;
constexpr int NUM_THREADS = 64 + 2 * 128;
constexpr uint32_t TMEM_COLS = 512;

enum { ERR_Q = 51, ERR_KV_FULL = 52, ERR_KV_EMPTY = 53, ERR_S = 54, ERR_P = 55, ERR_PV = 56 };

struct WindowParams {
  const int *pos, *count;
  const __nv_bfloat16* gate;  // first gate column of the projections, or null
  long long ldg;
  __nv_bfloat16* out;
  long long ldo;
  int T, H, G, dim, vdim, Smax, window, keep_first;
  float scale, sink;
  int* err;
};

using namespace xl_tc;

// DK: 64 or 128, query / key features rounded up; VD: 64 or 128, value features rounded up. Features past the real sizes are zero
// in the key and value tiles (TMA fills what lies outside the cache rows), so they add nothing.
template <int DK, int VD> struct WindowSmem {
  static constexpr int K_STAGES = DK == 64 ? 3 : 2;
  static constexpr int V_STAGES = VD == 64 ? 3 : 2;
  static constexpr int Q_BYTES = TILE_M * DK * 2;  // per tile: DK/64 blocks of (128 rows x 128 B)
  static constexpr int K_BYTES = BKV * DK * 2;
  static constexpr int V_BYTES = BKV * VD * 2;     // 2 blocks of VD/64 boxes of (64 rows x 128 B)
  static constexpr int TILE_BYTES = 2 * Q_BYTES + K_STAGES * K_BYTES + V_STAGES * V_BYTES;
  static constexpr int NEEDED = TILE_BYTES + 1024 /*alignment*/ + 256 /*barriers*/;
  // more than half of an SM's shared memory: two CTAs, each holding all of TMEM, never meet on an SM
  static constexpr int TOTAL = NEEDED > 120 * 1024 ? NEEDED : 120 * 1024;
};

template <int DK, int VD>
__global__ void __launch_bounds__(NUM_THREADS, 1)
    window_attn_tcgen05_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                               const __grid_constant__ CUtensorMap map_v, const WindowParams p) {
  using L = WindowSmem<DK, VD>;
  static_assert(L::TOTAL <= 227 * 1024, "shared memory");
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint8_t* sQ = smem;
  uint8_t* sK = smem + 2 * L::Q_BYTES;
  uint8_t* sV = sK + L::K_STAGES * L::K_BYTES;
  uint64_t* bars = (uint64_t*)(smem + L::TILE_BYTES);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;    // [3]
  uint64_t* k_empty = bars + 4;   // [3]
  uint64_t* v_full = bars + 7;    // [3]
  uint64_t* v_empty = bars + 10;  // [3]
  uint64_t* s_full = bars + 13;   // [2] per tile
  uint64_t* p_full = bars + 15;   // [2]
  uint64_t* pv_done = bars + 17;  // [2]
  uint32_t* tmem_base_slot = (uint32_t*)(bars + 19);
  volatile int* abort_flag = (volatile int*)(tmem_base_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = blockIdx.x, b = blockIdx.z, R = p.H / p.G;
  const int cnt = min(p.count[b], p.T), pos = p.pos[b];
  const long long rows = (long long)cnt * R;                              // real rows of this sequence and key / value head
  const long long f0 = (long long)(gridDim.y - 1 - blockIdx.y) * 2 * TILE_M;  // the blocks with the most keys first
  if (f0 >= rows || pos < 0 || pos + cnt > p.Smax) return;
  const int tiles = f0 + TILE_M < rows ? 2 : 1;
  const int p_first = pos + (int)(f0 / R), p_last = pos + (int)((min(rows, f0 + 2 * TILE_M) - 1) / R);
  // key blocks: those of the kept tokens that lie before every window of this CTA, then everything from there on; or, where
  // that takes no more blocks, simply all keys
  WindowRange seen = window_range(p_first, p.window, p.keep_first);
  int kept_blocks = (seen.kept + BKV - 1) / BKV;
  if (kept_blocks + (p_last - seen.first) / BKV >= p_last / BKV) {
    seen = {0, 0};
    kept_blocks = 0;
  }
  const int n_kv = kept_blocks + (p_last - seen.first) / BKV + 1;
  auto first_key = [&](int j) { return j < kept_blocks ? j * BKV : seen.first + (j - kept_blocks) * BKV; };

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < 3; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(&s_full[s], 1);
      mbar_init(&p_full[s], 4);
      mbar_init(&pv_done[s], 1);
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    tmem_alloc(tmem_base_slot, TMEM_COLS);
    tmem_relinquish();
  }
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem_base = *tmem_base_slot;

  if (warp == 0) {
    // lane 0: queries and key tiles, lane 1: value tiles; each waits only on its own ring
    if (lane < 2) {
      const bool for_k = lane == 0;
      if (for_k) {
        mbar_expect_tx(q_full, tiles * L::Q_BYTES);
        for (int m = 0; m < tiles; ++m)
#pragma unroll
          for (int kb = 0; kb < DK / 64; ++kb)
            tma_load_2d(sQ + m * L::Q_BYTES + kb * (TILE_M * 128), &map_q, q_full, kb * 64,
                        (int)((long long)(b * p.G + g) * p.T * R + f0) + m * TILE_M);
      }
      const int stages = for_k ? L::K_STAGES : L::V_STAGES;
      uint64_t* full = for_k ? k_full : v_full;
      uint64_t* empty = for_k ? k_empty : v_empty;
      bool ok = true;
      int issued = 0;
      for (int j = 0; j < n_kv && ok; ++j) {
        const int st = j % stages, row = (b * p.G + g) * p.Smax + first_key(j);
        if (j >= stages) {
          ok = mbar_wait(&empty[st], (uint32_t)(j / stages - 1) & 1u, abort_flag, p.err, ERR_KV_EMPTY);
          if (!ok) break;
        }
        if (for_k) {
          mbar_expect_tx(&full[st], L::K_BYTES);
#pragma unroll
          for (int kb = 0; kb < DK / 64; ++kb)
            tma_load_2d(sK + st * L::K_BYTES + kb * (BKV * 128), &map_k, &full[st], kb * 64, row);
        } else {
          mbar_expect_tx(&full[st], L::V_BYTES);
#pragma unroll
          for (int kk = 0; kk < BKV / 64; ++kk)
#pragma unroll
            for (int jn = 0; jn < VD / 64; ++jn)
              tma_load_2d(sV + st * L::V_BYTES + (kk * (VD / 64) + jn) * 8192, &map_v, &full[st], jn * 64, row + kk * 64);
        }
        issued = j + 1;
      }
      if (!ok || *abort_flag) {
        // loads in flight target this CTA's shared memory: give them a bounded time to land before the CTA ends
        if (for_k)
          for (uint32_t i = 0; i < MBAR_SPIN_LIMIT && !mbar_try_wait(q_full, 0); ++i) {}
        for (int j = max(0, issued - stages); j < issued; ++j)
          for (uint32_t i = 0; i < MBAR_SPIN_LIMIT && !mbar_try_wait(&full[j % stages], (uint32_t)(j / stages) & 1u); ++i) {}
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      // bf16 operands, fp32 accumulators. S: both K-major, N = BKV. O: A (P) from TMEM, B (V) MN-major (bit 16), N = VD.
      const uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BKV >> 3) << 17) | ((uint32_t)(TILE_M >> 4) << 24);
      const uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(VD >> 3) << 17) |
                               ((uint32_t)(TILE_M >> 4) << 24);
      bool ok = mbar_wait(q_full, 0, abort_flag, p.err, ERR_Q);
      auto issue_scores = [&](int j, int m) -> bool {
        const int st = j % L::K_STAGES;
        if (!mbar_wait(&k_full[st], (uint32_t)(j / L::K_STAGES) & 1u, abort_flag, p.err, ERR_KV_FULL)) return false;
        // the buffer still holds P of the previous block until its product has been taken
        if (j > 0 && !mbar_wait(&pv_done[m], (uint32_t)(j - 1) & 1u, abort_flag, p.err, ERR_PV)) return false;
        tcgen05_fence_after();
        const uint32_t q_addr = smem_u32(sQ + m * L::Q_BYTES), k_addr = smem_u32(sK + st * L::K_BYTES);
#pragma unroll
        for (int kb = 0; kb < DK / 64; ++kb)
#pragma unroll
          for (int k = 0; k < 64 / UMMA_K; ++k)
            tcgen05_mma_f16(tmem_base + m * BKV, make_smem_desc(q_addr + kb * (TILE_M * 128) + k * (UMMA_K * 2), 16),
                            make_smem_desc(k_addr + kb * (BKV * 128) + k * (UMMA_K * 2), 16), idesc_s, (kb | k) ? 1u : 0u);
        if (m == tiles - 1) tcgen05_commit(&k_empty[st]);
        tcgen05_commit(&s_full[m]);
        return true;
      };
      for (int m = 0; m < tiles && ok; ++m) ok = issue_scores(0, m);
      for (int j = 0; j < n_kv && ok; ++j) {
        const int st = j % L::V_STAGES;
        ok = mbar_wait(&v_full[st], (uint32_t)(j / L::V_STAGES) & 1u, abort_flag, p.err, ERR_KV_FULL);
        for (int m = 0; m < tiles && ok; ++m) {
          ok = mbar_wait(&p_full[m], (uint32_t)j & 1u, abort_flag, p.err, ERR_P);
          if (!ok) break;
          tcgen05_fence_after();
          const uint32_t v_addr = smem_u32(sV + st * L::V_BYTES);
          const uint32_t tmem_o = tmem_base + 2 * BKV + m * VD;
#pragma unroll
          for (int part = 0; part < 2; ++part)  // rounded weights, then their rounding errors
#pragma unroll
            for (int k = 0; k < BKV / UMMA_K; ++k)
              tcgen05_mma_f16_ts(tmem_o, tmem_base + m * BKV + part * (BKV / 2) + k * (UMMA_K / 2),
                                 make_smem_desc(v_addr + (k >> 2) * (VD / 64) * 8192 + (k & 3) * (UMMA_K * 128), 8192), idesc_o,
                                 (j | part | k) ? 1u : 0u);
          if (m == tiles - 1) tcgen05_commit(&v_empty[st]);
          tcgen05_commit(&pv_done[m]);
          if (j + 1 < n_kv) ok = issue_scores(j + 1, m);
        }
      }
    }
  } else if ((warp < 6 ? 0 : 1) < tiles) {
    const int m = warp < 6 ? 0 : 1;       // row tile of this warpgroup
    const int qtr = warp & 3;             // TMEM lane quarter this warp may access
    const int r = qtr * 32 + lane;        // row inside the tile
    const long long f = f0 + m * TILE_M + r;  // (token, head of the group)
    const int t = (int)(f / R), hh = (int)(f - (long long)t * R);
    const int qpos = pos + t;
    const int lo = window_range(qpos, p.window, 0).first;
    const uint32_t lane_base = (uint32_t)(qtr * 32) << 16;
    const uint32_t tmem_s = tmem_base + lane_base + m * BKV;
    const uint32_t tmem_o = tmem_base + lane_base + 2 * BKV + m * VD;
    const float c = p.scale * 1.4426950408889634f;
    float mx = p.sink / p.scale, l = p.sink == -INFINITY ? 0.f : 1.f;
    bool ok = true;
    for (int j = 0; j < n_kv && ok; ++j) {
      ok = __all_sync(0xffffffffu, mbar_wait(&s_full[m], (uint32_t)j & 1u, abort_flag, p.err, ERR_S));
      if (!ok) break;
      tcgen05_fence_after();
      float s[BKV];
#pragma unroll
      for (int ch = 0; ch < BKV / 32; ++ch) {
        uint32_t raw[32];
        tmem_ld_32x32b_x32(tmem_s + ch * 32, raw);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) s[ch * 32 + i] = __uint_as_float(raw[i]);
      }
      const int col0 = first_key(j), hi = j < kept_blocks ? seen.kept - 1 : qpos;
      if (col0 + BKV - 1 > hi || (col0 < lo && col0 + BKV > p.keep_first)) {
#pragma unroll
        for (int i = 0; i < BKV; ++i)
          if (col0 + i > hi || (col0 + i < lo && col0 + i >= p.keep_first)) s[i] = -INFINITY;
      }
      float m_blk = -INFINITY;
#pragma unroll
      for (int i = 0; i < BKV; ++i) m_blk = fmaxf(m_blk, s[i]);
      // the reference maximum moves (and O, l are rescaled) only when the exponent would exceed 2^8
      const bool move = m_blk > -INFINITY && (mx == -INFINITY || (m_blk - mx) * c > 8.f);
      const float m_new = move ? m_blk : mx;
      const float m_use = m_new == -INFINITY ? 0.f : m_new;  // a row without a visible key yet keeps weight 0
      const float alpha = (move && mx != -INFINITY) ? fast_exp2((mx - m_use) * c) : 1.f;
      const float mc = m_use * c;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < BKV; ++i) {
        s[i] = fast_exp2(fmaf(s[i], c, -mc));
        sum += s[i];
      }
      l = l * alpha + sum;
      mx = m_new;
      // the scores of block j are only computed after P V of block j - 1: O is at rest here
      if (j > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll 1
        for (int ch = 0; ch < VD / 32; ++ch) {
          uint32_t raw[32];
          tmem_ld_32x32b_x32(tmem_o + ch * 32, raw);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) raw[i] = __float_as_uint(__uint_as_float(raw[i]) * alpha);
          tmem_st_32x32b_x32(tmem_o + ch * 32, raw);
        }
      }
      store_split_weights<BKV>(tmem_s, s);
      tmem_st_wait();
      tcgen05_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[m]);
    }
    // ---- output: divided by the sum, gated -------------------------------------------------------------------------------
    ok = ok && __all_sync(0xffffffffu, mbar_wait(&pv_done[m], (uint32_t)(n_kv - 1) & 1u, abort_flag, p.err, ERR_PV));
    if (ok) {
      tcgen05_fence_after();
      const float inv = 1.f / l;
      const long long at = (long long)b * p.T + t, col = (long long)(g * R + hh) * p.vdim;
      const __nv_bfloat16* grow = p.gate ? p.gate + at * p.ldg + col : nullptr;
      __nv_bfloat16* orow = p.out + at * p.ldo + col;
#pragma unroll 1
      for (int ch = 0; ch < VD / 32; ++ch) {
        uint32_t raw[32];
        tmem_ld_32x32b_x32(tmem_o + ch * 32, raw);
        tmem_ld_wait();
        if (f < rows) {
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int c0 = ch * 32 + q * 8;
            if (c0 < p.vdim) {
              float v[8];
#pragma unroll
              for (int e = 0; e < 8; ++e) v[e] = __uint_as_float(raw[q * 8 + e]) * inv;
              if (grow) {
                float gt[8];
                xl_load16<__nv_bfloat16>(grow + c0, gt);
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] *= __fdividef(1.f, 1.f + __expf(-gt[e]));
              }
              *(uint4*)(orow + c0) = pack8_16bit(v, false);
            }
          }
        }
      }
    }
  }

  // ---- teardown: every role arrives here, also after an abort --------------------------------------------------------
  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

template <int DK, int VD>
int launch(const void* qn, const void* kc, const void* vc, const WindowParams& p, int B, cudaStream_t s) {
  using L = WindowSmem<DK, VD>;
  CUtensorMap mq, mk, mv;
  int r = make_map_bf16(&mq, qn, (long long)B * p.T * p.H, p.dim, p.dim, TILE_M);
  if (r) return r;
  r = make_map_bf16(&mk, kc, (long long)B * p.G * p.Smax, p.dim, p.dim, BKV);
  if (r) return r;
  r = make_map_bf16(&mv, vc, (long long)B * p.G * p.Smax, p.vdim, p.vdim, 64);
  if (r) return r;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e =
        cudaFuncSetAttribute(window_attn_tcgen05_kernel<DK, VD>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const long long rows = (long long)p.T * (p.H / p.G);
  const dim3 grid(p.G, (unsigned)((rows + 2 * TILE_M - 1) / (2 * TILE_M)), B);
  window_attn_tcgen05_kernel<DK, VD><<<grid, NUM_THREADS, L::TOTAL, s>>>(mq, mk, mv, p);
  return (int)cudaGetLastError();
}

}  // namespace

// qn (B, G, T, H/G, dim) bf16, normalised; caches as in attention_window.cu with the portion's keys and values in place; gate:
// first gate column of the projections (row stride ldg), or null; out (B*T, ldo). dim, vdim multiples of 8 and at most 128; ldg,
// ldo multiples of 8; all pointers 16-byte aligned. Rows past count[b] are not written. err: device int for the code of a wait
// that gave up. Returns 0, a CUDA error code, or a negative value for arguments this kernel does not take.
XL_API int xl_window_attn_tcgen05(const void* qn, const void* kc, const void* vc, const void* gate, long long ldg, void* out,
                                  long long ldo, const int* pos, const int* count, int B, int T, int H, int G, int dim, int vdim,
                                  int Smax, int window, int keep_first, float scale, float sink, int* err, cudaStream_t s) {
  if (B < 1 || B > 65535 || T < 1 || G < 1 || H < 1 || H % G || Smax < 1 || window < 0 || keep_first < 0) return -1;
  if (dim < 8 || dim > 128 || dim % 8 || vdim < 8 || vdim > 128 || vdim % 8 || ldo % 8 || ldo < (long long)H * vdim ||
      (gate && (ldg % 8 || ldg < (long long)H * vdim)))
    return -1;
  if ((((uintptr_t)qn) | ((uintptr_t)kc) | ((uintptr_t)vc) | ((uintptr_t)gate) | ((uintptr_t)out)) & 15) return -1;
  if (!(scale > 0.f) || (long long)B * G * Smax > 0x7fffffffLL - 2 * BKV || (long long)B * T * H > 0x7fffffffLL - 4 * TILE_M ||
      ((long long)T * (H / G) + 2 * TILE_M - 1) / (2 * TILE_M) > 65535)
    return -1;
  WindowParams p;
  p.pos = pos; p.count = count; p.gate = (const __nv_bfloat16*)gate; p.ldg = ldg; p.out = (__nv_bfloat16*)out; p.ldo = ldo;
  p.T = T; p.H = H; p.G = G; p.dim = dim; p.vdim = vdim; p.Smax = Smax; p.window = window; p.keep_first = keep_first;
  p.scale = scale; p.sink = sink; p.err = err;
  if (dim <= 64) return vdim <= 64 ? launch<64, 64>(qn, kc, vc, p, B, s) : launch<64, 128>(qn, kc, vc, p, B, s);
  return vdim <= 64 ? launch<128, 64>(qn, kc, vc, p, B, s) : launch<128, 128>(qn, kc, vc, p, B, s);
}
