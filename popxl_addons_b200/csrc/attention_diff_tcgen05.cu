// Differential attention of a portion of tokens against the key / value cache on the 5th-generation tensor cores (tcgen05),
// bf16. Same mathematics and layouts as attention_diff.cu: two query / key maps per head over shared values, causal, chunked
// visibility, o = a_1 - lambda a_2 divided by its root mean square.
//
// One CTA owns 128 query rows of one head and both of its maps, and walks the visible keys in blocks of 128:
//   warp 0       TMA producer : the query tiles of both maps once, key tiles (block, map) and value tiles through two rings
//   warp 1       MMA issuer   : S_m = Q_m K_m^T into TMEM, then O_m += P_m V, the two maps taking turns, so that the softmax
//                               of one map runs under the products of the other
//   warps 2..5   softmax of map 1, warps 6..9 of map 2: one thread per query row; running maximum and sum in fp32, lazy
//                               rescaling of O_m in TMEM
// P replaces S in TMEM (the product takes its A operand from there) as two bf16 numbers per weight, value and rounding error:
// the two maps' results nearly cancel in a_1 - lambda a_2, and weights rounded to bf16 would be the largest error there.
//
// TMEM columns: [0, 128) S_1 / P_1, [128, 256) S_2 / P_2 (the upper half of each holds the rounding errors),
// [256, 256 + VD) O_1, [256 + VD, 256 + 2 VD) O_2. One CTA per SM. Every wait is bounded (see tcgen05.cuh).
#include "tcgen05.cuh"

namespace {

constexpr int BLOCK_Q = 128;
constexpr int BKV = 128;
constexpr int UMMA_K = 16;
constexpr int V_STAGES = 2;
constexpr int NUM_THREADS = 64 + 2 * 128;
constexpr uint32_t TMEM_COLS = 512;

enum { ERR_Q = 41, ERR_KV_FULL = 42, ERR_KV_EMPTY = 43, ERR_S = 44, ERR_P = 45, ERR_PV = 46 };

struct DiffParams {
  const int *pos, *count;
  const float* lam;
  __nv_bfloat16* out;
  long long ldo;
  int T, H, G, dim, vdim, Smax, chunk;
  float scale, eps, out_scale;
  int* err;
};

using namespace xl_tc;

// DK: 64 or 128, query / key features per map rounded up; VD: 64 or 128, value features rounded up. Features past the real
// sizes are zero in the key and value tiles (TMA fills what lies outside the cache rows), so they add nothing.
template <int DK, int VD> struct DiffSmem {
  static constexpr int K_STAGES = DK == 64 ? 4 : 3;  // tiles of one map
  static constexpr int Q_BYTES = BLOCK_Q * DK * 2;   // per map: DK/64 blocks of (128 rows x 128 B)
  static constexpr int K_BYTES = BKV * DK * 2;
  static constexpr int V_BYTES = BKV * VD * 2;       // 2 blocks of VD/64 boxes of (64 rows x 128 B)
  static constexpr int TILE_BYTES = 2 * Q_BYTES + K_STAGES * K_BYTES + V_STAGES * V_BYTES;
  static constexpr int NEEDED = TILE_BYTES + 1024 /*alignment*/ + 256 /*barriers*/ + 512 /*sums of map 2*/;
  // more than half of an SM's shared memory: two CTAs, each holding all of TMEM, never meet on an SM
  static constexpr int TOTAL = NEEDED > 120 * 1024 ? NEEDED : 120 * 1024;
};

template <int DK, int VD>
__global__ void __launch_bounds__(NUM_THREADS, 1)
    diff_attn_tcgen05_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                             const __grid_constant__ CUtensorMap map_v, const DiffParams p) {
  using L = DiffSmem<DK, VD>;
  static_assert(L::TOTAL <= 227 * 1024, "shared memory");
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint8_t* sQ = smem;
  uint8_t* sK = smem + 2 * L::Q_BYTES;
  uint8_t* sV = sK + L::K_STAGES * L::K_BYTES;
  uint64_t* bars = (uint64_t*)(smem + L::TILE_BYTES);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;    // [4]
  uint64_t* k_empty = bars + 5;   // [4]
  uint64_t* v_full = bars + 9;    // [2]
  uint64_t* v_empty = bars + 11;  // [2]
  uint64_t* s_full = bars + 13;   // [2] per map
  uint64_t* p_full = bars + 15;   // [2]
  uint64_t* pv_done = bars + 17;  // [2]
  uint64_t* sum_ready = bars + 19;
  uint32_t* tmem_base_slot = (uint32_t*)(bars + 20);
  volatile int* abort_flag = (volatile int*)(tmem_base_slot + 1);
  float* sum2 = (float*)(smem + L::TILE_BYTES + 256);  // [128] 1 / l of map 2

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, b = blockIdx.z, g = h / (p.H / p.G);
  const int t0 = (int)(gridDim.y - 1 - blockIdx.y) * BLOCK_Q;  // the blocks with the most keys first
  const int cnt = min(p.count[b], p.T), pos = p.pos[b];
  if (t0 >= cnt || pos < 0 || pos + cnt > p.Smax) return;
  const int p_first = pos + t0, p_last = pos + min(cnt, t0 + BLOCK_Q) - 1;
  const int key0 = p.chunk > 0 ? (p_first / p.chunk) * p.chunk : 0;  // first key that any row of this block may see
  const int n_kv = (p_last - key0) / BKV + 1;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < 4; ++s) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(&v_full[s], 1);
      mbar_init(&v_empty[s], 1);
      mbar_init(&s_full[s], 1);
      mbar_init(&p_full[s], 4);
      mbar_init(&pv_done[s], 1);
    }
    mbar_init(sum_ready, 4);
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
        mbar_expect_tx(q_full, 2 * L::Q_BYTES);
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
          for (int kb = 0; kb < DK / 64; ++kb)
            tma_load_2d(sQ + m * L::Q_BYTES + kb * (BLOCK_Q * 128), &map_q, q_full, (h * 2 + m) * p.dim + kb * 64,
                        b * p.T + t0);
      }
      const int n_tiles = for_k ? 2 * n_kv : n_kv;
      const int stages = for_k ? L::K_STAGES : V_STAGES;
      uint64_t* full = for_k ? k_full : v_full;
      uint64_t* empty = for_k ? k_empty : v_empty;
      bool ok = true;
      int issued = 0;
      for (int i = 0; i < n_tiles && ok; ++i) {
        const int st = i % stages;
        if (i >= stages) {
          ok = mbar_wait(&empty[st], (uint32_t)(i / stages - 1) & 1u, abort_flag, p.err, ERR_KV_EMPTY);
          if (!ok) break;
        }
        if (for_k) {
          const int j = i >> 1, m = i & 1;
          mbar_expect_tx(&full[st], L::K_BYTES);
          const int row = ((b * p.G + g) * 2 + m) * p.Smax + key0 + j * BKV;
#pragma unroll
          for (int kb = 0; kb < DK / 64; ++kb)
            tma_load_2d(sK + st * L::K_BYTES + kb * (BKV * 128), &map_k, &full[st], kb * 64, row);
        } else {
          mbar_expect_tx(&full[st], L::V_BYTES);
          const int row = (b * p.G + g) * p.Smax + key0 + i * BKV;
#pragma unroll
          for (int kk = 0; kk < BKV / 64; ++kk)
#pragma unroll
            for (int jn = 0; jn < VD / 64; ++jn)
              tma_load_2d(sV + st * L::V_BYTES + (kk * (VD / 64) + jn) * 8192, &map_v, &full[st], jn * 64, row + kk * 64);
        }
        issued = i + 1;
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
      const uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BKV >> 3) << 17) | ((uint32_t)(BLOCK_Q >> 4) << 24);
      const uint32_t idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(VD >> 3) << 17) |
                               ((uint32_t)(BLOCK_Q >> 4) << 24);
      bool ok = mbar_wait(q_full, 0, abort_flag, p.err, ERR_Q);
      auto issue_scores = [&](int j, int m) -> bool {
        const int i = 2 * j + m, st = i % L::K_STAGES;
        if (!mbar_wait(&k_full[st], (uint32_t)(i / L::K_STAGES) & 1u, abort_flag, p.err, ERR_KV_FULL)) return false;
        // the buffer still holds P of the previous block until its product has been taken
        if (j > 0 && !mbar_wait(&pv_done[m], (uint32_t)(j - 1) & 1u, abort_flag, p.err, ERR_PV)) return false;
        tcgen05_fence_after();
        const uint32_t q_addr = smem_u32(sQ + m * L::Q_BYTES), k_addr = smem_u32(sK + st * L::K_BYTES);
#pragma unroll
        for (int kb = 0; kb < DK / 64; ++kb)
#pragma unroll
          for (int k = 0; k < 64 / UMMA_K; ++k)
            tcgen05_mma_f16(tmem_base + m * BKV, make_smem_desc(q_addr + kb * (BLOCK_Q * 128) + k * (UMMA_K * 2), 16),
                            make_smem_desc(k_addr + kb * (BKV * 128) + k * (UMMA_K * 2), 16), idesc_s, (kb | k) ? 1u : 0u);
        tcgen05_commit(&k_empty[st]);
        tcgen05_commit(&s_full[m]);
        return true;
      };
      ok = ok && issue_scores(0, 0) && issue_scores(0, 1);
      for (int j = 0; j < n_kv && ok; ++j) {
        const int st = j % V_STAGES;
        ok = mbar_wait(&v_full[st], (uint32_t)(j / V_STAGES) & 1u, abort_flag, p.err, ERR_KV_FULL);
        for (int m = 0; m < 2 && ok; ++m) {
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
          if (m == 1) tcgen05_commit(&v_empty[st]);
          tcgen05_commit(&pv_done[m]);
          if (j + 1 < n_kv) ok = issue_scores(j + 1, m);
        }
      }
    }
  } else {
    const int m = warp < 6 ? 0 : 1;       // map of this warpgroup
    const int qtr = warp & 3;             // TMEM lane quarter this warp may access
    const int r = qtr * 32 + lane;        // query row inside the block
    const int qpos = p_first + r;         // its position
    const int lo = p.chunk > 0 ? (qpos / p.chunk) * p.chunk : 0;
    const uint32_t lane_base = (uint32_t)(qtr * 32) << 16;
    const uint32_t tmem_s = tmem_base + lane_base + m * BKV;
    const uint32_t tmem_o = tmem_base + lane_base + 2 * BKV + m * VD;
    const float c = p.scale * 1.4426950408889634f;
    float mx = -INFINITY, l = 0.f;
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
      const int col0 = key0 + j * BKV;
      if (col0 < lo || col0 + BKV - 1 > qpos) {
#pragma unroll
        for (int i = 0; i < BKV; ++i)
          if (col0 + i < lo || col0 + i > qpos) s[i] = -INFINITY;
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
    // ---- combination: map 2 hands over its sums, map 1's warps read both accumulators of their rows ---------------------
    if (m == 1) {
      sum2[r] = l > 0.f ? 1.f / l : 0.f;
      __syncwarp();
      if (lane == 0) mbar_arrive(sum_ready);
    } else {
      const uint32_t last = (uint32_t)(n_kv - 1) & 1u;
      ok = ok && __all_sync(0xffffffffu, mbar_wait(&pv_done[0], last, abort_flag, p.err, ERR_PV) &&
                                             mbar_wait(&pv_done[1], last, abort_flag, p.err, ERR_PV) &&
                                             mbar_wait(sum_ready, 0, abort_flag, p.err, ERR_PV));
      if (ok) {
        tcgen05_fence_after();
        const float i1 = l > 0.f ? 1.f / l : 0.f, i2 = *p.lam * sum2[r];
        float ss = 0.f;
#pragma unroll 1
        for (int ch = 0; ch < VD / 32; ++ch) {
          uint32_t r1[32], r2[32];
          tmem_ld_32x32b_x32(tmem_o + ch * 32, r1);
          tmem_ld_32x32b_x32(tmem_o + VD + ch * 32, r2);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float v = __uint_as_float(r1[i]) * i1 - __uint_as_float(r2[i]) * i2;
            ss += v * v;  // columns past vdim are zero
          }
        }
        const float f = p.out_scale / sqrtf(ss / p.vdim + p.eps);
        __nv_bfloat16* orow = p.out + ((long long)b * p.T + t0 + r) * p.ldo + (long long)h * p.vdim;
#pragma unroll 1
        for (int ch = 0; ch < VD / 32; ++ch) {
          uint32_t r1[32], r2[32];
          tmem_ld_32x32b_x32(tmem_o + ch * 32, r1);
          tmem_ld_32x32b_x32(tmem_o + VD + ch * 32, r2);
          tmem_ld_wait();
          if (t0 + r < cnt) {
#pragma unroll
            for (int q = 0; q < 4; ++q) {
              float v[8];
#pragma unroll
              for (int e = 0; e < 8; ++e)
                v[e] = (__uint_as_float(r1[q * 8 + e]) * i1 - __uint_as_float(r2[q * 8 + e]) * i2) * f;
              if (ch * 32 + q * 8 < p.vdim) *(uint4*)(orow + ch * 32 + q * 8) = pack8_16bit(v, false);
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
int launch(const void* q, long long ldq, const void* kc, const void* vc, const DiffParams& p, int B, cudaStream_t s) {
  using L = DiffSmem<DK, VD>;
  CUtensorMap mq, mk, mv;
  int r = make_map_bf16(&mq, q, (long long)B * p.T, ldq, ldq, BLOCK_Q);
  if (r) return r;
  r = make_map_bf16(&mk, kc, (long long)B * p.G * 2 * p.Smax, p.dim, p.dim, BKV);
  if (r) return r;
  r = make_map_bf16(&mv, vc, (long long)B * p.G * p.Smax, p.vdim, p.vdim, 64);
  if (r) return r;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e =
        cudaFuncSetAttribute(diff_attn_tcgen05_kernel<DK, VD>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const dim3 grid(p.H, (p.T + BLOCK_Q - 1) / BLOCK_Q, B);
  diff_attn_tcgen05_kernel<DK, VD><<<grid, NUM_THREADS, L::TOTAL, s>>>(mq, mk, mv, p);
  return (int)cudaGetLastError();
}

}  // namespace

// q: (B*T, ldq) bf16, head h and map m in columns [(2h + m) dim, ...), already rotated; caches as in attention_diff.cu with the
// portion's keys and values in place; out (B*T, ldo). dim, vdim multiples of 8 and at most 128; ldq, ldo multiples of 8;
// q, kc, vc, out 16-byte aligned. Rows past count[b] are not written. err: device int for the code of a wait that gave up.
// Returns 0, a CUDA error code, or a negative value for arguments this kernel does not take.
XL_API int xl_diff_attn_tcgen05(const void* q, long long ldq, const void* kc, const void* vc, void* out, long long ldo,
                                const int* pos, const int* count, const float* lam, int B, int T, int H, int G, int dim, int vdim,
                                int Smax, int chunk, float scale, float eps, float out_scale, int* err, cudaStream_t s) {
  if (B < 1 || B > 65535 || T < 1 || (T + BLOCK_Q - 1) / BLOCK_Q > 65535 || G < 1 || H < 1 || H % G || Smax < 1 || chunk < 0)
    return -1;
  if (dim < 8 || dim > 128 || dim % 8 || vdim < 8 || vdim > 128 || vdim % 8 || ldq % 8 || ldo % 8 || ldq < (long long)H * 2 * dim ||
      ldo < (long long)H * vdim)
    return -1;
  if ((((uintptr_t)q) & 15) || (((uintptr_t)kc) & 15) || (((uintptr_t)vc) & 15) || (((uintptr_t)out) & 15) || !(scale > 0.f)) return -1;
  if ((long long)B * G * 2 * Smax > 0x7fffffffLL - 2 * BKV) return -1;
  DiffParams p;
  p.pos = pos; p.count = count; p.lam = lam; p.out = (__nv_bfloat16*)out; p.ldo = ldo; p.T = T; p.H = H; p.G = G; p.dim = dim;
  p.vdim = vdim; p.Smax = Smax; p.chunk = chunk; p.scale = scale; p.eps = eps; p.out_scale = out_scale; p.err = err;
  if (dim <= 64) return vdim <= 64 ? launch<64, 64>(q, ldq, kc, vc, p, B, s) : launch<64, 128>(q, ldq, kc, vc, p, B, s);
  return vdim <= 64 ? launch<128, 64>(q, ldq, kc, vc, p, B, s) : launch<128, 128>(q, ldq, kc, vc, p, B, s);
}
