// Attention of a packed prompt step of the layered decoder models, on the 5th-generation tensor cores.  Three kinds of layers:
// sliding-window latent attention, (BIAS) causal grouped-query attention with a learned bias per head and distance, and (CAPPED)
// windowed or chunked grouped-query attention with capped scores and an optional sink.
//
// Queries [T, H, dim + rot], unrotated keys [K, H, dim] and values [K, H, vdim] (one packed matrix), one rotated key part
// [K, rot] shared by all heads.  Every size that is a multiple of eight is taken as it is: operand panels are 64 columns
// wide and the copy engine zero-fills past dim, rot and vdim.
//
// One CTA per (256 queries of one sequence, head): two 128-query tiles share every key / value block and ping-pong on one
// MMA issuer (the scheme of attn_fwd2_kernel in attention.cu):
//   warps 0-3 / 4-7  softmax of tile A / B, one query row per thread: scores from tensor memory, window and causal mask on
//                    the edge blocks, lazy rescale of the accumulator, bf16 weights written back over the scores
//   warp 8           TMA: lane 0 queries and the key ring, lane 1 the value ring
//   warp 9           MMA issuer: S = Q K^T over the unrotated and rotated panels, O += P V with P in tensor memory
// Only key blocks that some query of a tile can see are visited.  The epilogue divides by the softmax sum and applies the
// layer's output gate.
//
// BIAS: keys and values come straight from the cache (key index = row * capacity + position), there is no rotated part, a
// query's scores carry its temperature and the gate is one number per head.  Blocks whose distances all lie in one bucket
// add a constant; the others (those near the diagonal) read the bias per element, lanes at consecutive distances.
//
// CAPPED: keys and values come from the step's key stream, there is neither a rotated part nor a gate.  A tile lies inside one chunk,
// so a chunk is nothing but the first key of its tiles.  Scores are cap tanh(score / cap): a polynomial on the FMA pipe as long as
// every score of a warp's columns is well below the cap, exponential and reciprocal otherwise.
//
// KEPT: CAPPED with the first keys of a sequence visible beside the window: their blocks come in front of the window's when there is a gap
// between the two, and are the first of one range otherwise.
//
// BOUNDED: CAPPED with a cap that is not large; SMALL: KEPT with scores that are small without a cap.  The softmax needs no running maximum and takes its columns as they come, and a query
// row is shared by two threads: sixteen softmax warps, each with half of a block's columns and its weights over its own half of the
// scores.
#include <cuda.h>

#include <type_traits>

#include <type_traits>

#include "common.cuh"
#include "softmax_math.cuh"

namespace b200 {

constexpr int LA_BM = 128;
constexpr int LA_QPANEL = LA_BM * 128;   // 128 rows x 64 bf16
constexpr int LA_MAX_STAGES = 3;

struct LatentAttnParams {
  int H, dim, rot, vdim, window;
  int pn, pr, pv;               // 64-column panels of the unrotated, rotated and value parts
  int kst, vst;                 // ring stages
  float scale_log2;
  const int4* tiles;            // {first query token, queries (1..256), stream index of the first query, first key of its sequence}
  const __nv_bfloat16* gate;    // [T, ld_gate], head h at column h * vdim
  __nv_bfloat16* out;           // [T, ld_out]
  int ld_gate, ld_out;
  int* err;
  // BIAS
  int group;                    // query heads per key / value head
  const float* bias;            // [H, ld_bias] in log2 units; distance d at column LA_BIAS_LEAD + d
  const int* bucket;            // [bias_len] bucket of each distance; the last entry holds for all farther ones
  int bias_len, ld_bias;
  int temp_every;               // 0: no temperature
  float temp_coef, gate_mult;
  // CAPPED (and `group`)
  const float* sink;            // [H] natural-log units; null: none
  int capped;                   // scores are capped
  float cap_log2, cap_exp;      // cap in log2 units; exponent of e^(2 score / cap) per raw score, log2 units
  int keep;                     // keys of a sequence that stay visible beside the window
  float cap_poly[3], poly_max;  // capped log2 score = raw * polynomial(raw^2) for |raw| <= poly_max
};
enum AttnKind { LATENT = 0, BIAS = 1, CAPPED = 2, BOUNDED = 3, KEPT = 4, SMALL = 5 };
__host__ __device__ constexpr bool la_bounded(int kind) { return kind == BOUNDED || kind == SMALL; }     // no running maximum
__host__ __device__ constexpr bool la_keeps(int kind) { return kind == KEPT || kind == SMALL; }
__host__ __device__ constexpr int la_softmax_warps(int kind) { return la_bounded(kind) ? 16 : 8; }
__host__ __device__ constexpr int la_threads(int kind) { return 32 * (la_softmax_warps(kind) + 4); }
// Columns in front of distance 0 and behind the last stored one (repeating the values there): a block's accesses need no clamps.
constexpr int LA_BIAS_LEAD = 256, LA_BIAS_TAIL = 256;

// The wait names the registers of the load: nothing that reads them moves in front of it.
__device__ __forceinline__ void tmem_ld_wait(uint32_t (&v)[32]) {
  asm volatile("tcgen05.wait::ld.sync.aligned;"
               : "+r"(v[0]), "+r"(v[1]), "+r"(v[2]), "+r"(v[3]), "+r"(v[4]), "+r"(v[5]), "+r"(v[6]), "+r"(v[7]), "+r"(v[8]), "+r"(v[9]), "+r"(v[10]),
                 "+r"(v[11]), "+r"(v[12]), "+r"(v[13]), "+r"(v[14]), "+r"(v[15]), "+r"(v[16]), "+r"(v[17]), "+r"(v[18]), "+r"(v[19]), "+r"(v[20]),
                 "+r"(v[21]), "+r"(v[22]), "+r"(v[23]), "+r"(v[24]), "+r"(v[25]), "+r"(v[26]), "+r"(v[27]), "+r"(v[28]), "+r"(v[29]), "+r"(v[30]),
                 "+r"(v[31])::"memory");
}
// Largest magnitude among N values.
template <int N>
__device__ __forceinline__ float max_abs(const float (&v)[N]) {
  float a4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < N; i += 8) {
    a4[0] = fmax3(a4[0], fabsf(v[i]), fabsf(v[i + 1]));
    a4[1] = fmax3(a4[1], fabsf(v[i + 2]), fabsf(v[i + 3]));
    a4[2] = fmax3(a4[2], fabsf(v[i + 4]), fabsf(v[i + 5]));
    a4[3] = fmax3(a4[3], fabsf(v[i + 6]), fabsf(v[i + 7]));
  }
  return fmaxf(fmaxf(a4[0], a4[1]), fmaxf(a4[2], a4[3]));
}
// Raw score -> capped score in log2 units: small raw scores (two at a time) / any.
__device__ __forceinline__ float2 cap_small(float2 x, const LatentAttnParams& p) {
  const float2 u = fmul2(x, x);
  return fmul2(ffma2(ffma2(make_float2(p.cap_poly[2], p.cap_poly[2]), u, make_float2(p.cap_poly[1], p.cap_poly[1])), u,
                     make_float2(p.cap_poly[0], p.cap_poly[0])), x);
}
__device__ __forceinline__ float cap_any(float x, const LatentAttnParams& p) {
  return p.cap_log2 - 2.f * p.cap_log2 * rcp_approx(1.f + ex2_approx(x * p.cap_exp));
}

// Position in a ring of `n` stages: stage index and the parity of the pass over the ring.
struct RingPos {
  int s = 0;
  uint32_t ph = 0;
  __device__ __forceinline__ void next(int n) {
    if (++s == n) { s = 0; ph ^= 1; }
  }
};

struct LatentAttnBars {
  uint64_t q_full[2];
  uint64_t k_full[LA_MAX_STAGES], k_empty[LA_MAX_STAGES], v_full[LA_MAX_STAGES], v_empty[LA_MAX_STAGES];
  uint64_t s_full[2], p_ready[2], o_final[2];
  uint32_t tmem_slot;
  int abort_flag;
};

// SN, SR: 16-column MMA steps of the unrotated and rotated parts, known at compile time for common sizes (a block's score
// product is then a straight line of MMAs: the issuing thread's address arithmetic would otherwise pace the whole block);
// 0: read from the parameters.
template <int BN, int SN, int SR, int KIND = LATENT>
__global__ void __launch_bounds__(la_threads(KIND), 1)
latent_attn_kernel(const __grid_constant__ CUtensorMap tmQn, const __grid_constant__ CUtensorMap tmQr,
                   const __grid_constant__ CUtensorMap tmKn, const __grid_constant__ CUtensorMap tmKr,
                   const __grid_constant__ CUtensorMap tmV, const LatentAttnParams p) {
  constexpr int KPANEL = BN * 128;
  constexpr uint32_t IDESC_S = make_idesc_bf16(LA_BM, BN, 0, 0);
  constexpr int O_COL = 2 * BN, O_WIDTH = (512 - 2 * BN) / 2;
  constexpr float RESCALE_THRESHOLD = 8.f;   // log2 units
  constexpr int WARPS = la_softmax_warps(KIND), SPLIT = WARPS / 8;   // SPLIT: threads per query row

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int pn = SN ? (SN + 3) / 4 : p.pn, pr = SN ? (SR + 3) / 4 : p.pr, kp = pn + pr;
  const int q_bytes = kp * LA_QPANEL, k_bytes = kp * KPANEL, v_bytes = p.pv * KPANEL;
  LatentAttnBars* bars = reinterpret_cast<LatentAttnBars*>(smem);   // in front: offsets that do not depend on the sizes
  uint8_t* sQ = smem + 1024;                // tile A, tile B
  uint8_t* sK = sQ + 2 * q_bytes;
  uint8_t* sV = sK + p.kst * k_bytes;
  volatile int* abort_flag = &bars->abort_flag;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, hk = KIND != LATENT ? h / p.group : h;
  const int4 tile = p.tiles[blockIdx.y];
  const int q0 = tile.x, nrows = tile.y, s0 = tile.z, kbase = tile.w;
  int kstart = max(kbase, s0 - p.window + 1);
  // key blocks [jb, je) of both tiles: nkb blocks of kept keys, the others counted from kstart
  int nkb = 0;
  if constexpr (la_keeps(KIND)) {
    if (p.keep > 0) {
      nkb = (p.keep + BN - 1) / BN;
      if (kstart - kbase <= nkb * BN) {
        nkb = 0;
        kstart = kbase;
      }
    }
  }
  const bool keeps = la_keeps(KIND) && p.keep > 0;
  const int last_a = min(LA_BM, nrows) - 1, last_b = nrows - 1;
  const int je0 = nkb + (s0 + last_a - kstart) / BN + 1;
  const int jb1 = nrows > LA_BM && !keeps ? (max(kbase, s0 + LA_BM - p.window + 1) - kstart) / BN : 0;
  const int je1 = nrows > LA_BM ? nkb + (s0 + last_b - kstart) / BN + 1 : 0;
  const int nmax = max(je0, je1);
  auto block_key = [&](int j) { return la_keeps(KIND) ? (j < nkb ? kbase + j * BN : kstart + (j - nkb) * BN) : kstart + j * BN; };   // first key of a block

  auto load_q = [&](int x) {
    mbar_expect_tx(&bars->q_full[x], q_bytes);
    for (int c = 0; c < pn; ++c)
      tma_load_3d(sQ + x * q_bytes + c * LA_QPANEL, &tmQn, &bars->q_full[x], c * 64, q0 + x * LA_BM, h);
    for (int c = 0; c < pr; ++c)
      tma_load_3d(sQ + x * q_bytes + (pn + c) * LA_QPANEL, &tmQr, &bars->q_full[x], c * 64, q0 + x * LA_BM, h);
  };
  auto load_k = [&](int j, int s) {
    mbar_expect_tx(&bars->k_full[s], k_bytes);
    for (int c = 0; c < pn; ++c) tma_load_3d(sK + s * k_bytes + c * KPANEL, &tmKn, &bars->k_full[s], c * 64, block_key(j), hk);
    for (int c = 0; c < pr; ++c)
      tma_load_2d(sK + s * k_bytes + (pn + c) * KPANEL, &tmKr, &bars->k_full[s], c * 64, kstart + j * BN);
  };

  // the TMA thread sets up the barriers and requests the queries and the first key block before the CTA-wide sync
  if (threadIdx.x == 32 * WARPS) {
    tma_prefetch_desc(&tmQn);
    tma_prefetch_desc(&tmKn);
    if constexpr (KIND == LATENT) {
      tma_prefetch_desc(&tmQr);
      tma_prefetch_desc(&tmKr);
    }
    tma_prefetch_desc(&tmV);
    for (int i = 0; i < LA_MAX_STAGES; ++i) {
      mbar_init(&bars->k_full[i], 1);
      mbar_init(&bars->k_empty[i], 1);
      mbar_init(&bars->v_full[i], 1);
      mbar_init(&bars->v_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->q_full[i], 1);
      mbar_init(&bars->s_full[i], 1);
      mbar_init(&bars->p_ready[i], 4 * SPLIT);
      mbar_init(&bars->o_final[i], 1);
    }
    bars->abort_flag = 0;
    fence_barrier_init();
    fence_proxy_async_smem();
    load_q(0);            // rows past the sequence are other tokens or zero; they are never stored
    load_k(0, 0);
    load_q(1);
  }
  if (warp == WARPS + 1) {
    tmem_alloc(&bars->tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = bars->tmem_slot;

  if (warp >= WARPS) {
    if constexpr (SPLIT == 1) asm volatile("setmaxnreg.dec.sync.aligned.u32 72;");
    if (warp == WARPS) {
      if (lane == 0) {
        int issued = 1;
        RingPos k;
        k.next(p.kst);
        for (int j = 1; j < nmax; ++j, k.next(p.kst)) {
          if (!mbar_wait(&bars->k_empty[k.s], k.ph ^ 1, abort_flag, p.err, ERR_WAIT_ATTN)) break;
          load_k(j, k.s);
          issued = j + 1;
        }
        // every issued load must land before the CTA exits
        unsigned long long t0 = globaltimer_ns();
        while (!(mbar_try_wait(&bars->q_full[0], 0) && mbar_try_wait(&bars->q_full[1], 0)) && globaltimer_ns() - t0 < WAIT_LIMIT_NS) {}
        for (int j = max(0, issued - p.kst); j < issued; ++j) {
          t0 = globaltimer_ns();
          while (!mbar_try_wait(&bars->k_full[j % p.kst], (j / p.kst) & 1) && globaltimer_ns() - t0 < WAIT_LIMIT_NS) {}
        }
      } else if (lane == 1) {
        int issued = 0;
        RingPos v;
        for (int j = 0; j < nmax; ++j, v.next(p.vst)) {
          const int s = v.s;
          if (!mbar_wait(&bars->v_empty[s], v.ph ^ 1, abort_flag, p.err, ERR_WAIT_ATTN)) break;
          mbar_expect_tx(&bars->v_full[s], v_bytes);
          for (int c = 0; c < p.pv; ++c)
            tma_load_3d(sV + s * v_bytes + c * KPANEL, &tmV, &bars->v_full[s], c * 64, block_key(j), hk);
          issued = j + 1;
        }
        for (int j = max(0, issued - p.vst); j < issued; ++j) {
          const unsigned long long t0 = globaltimer_ns();
          while (!mbar_try_wait(&bars->v_full[j % p.vst], (j / p.vst) & 1) && globaltimer_ns() - t0 < WAIT_LIMIT_NS) {}
        }
      }
    } else if (KIND == LATENT && warp >= WARPS + 2) {
      // bring the CTA's gate rows into L2 while the blocks are processed
      const int lines = (2 * p.vdim + 127) / 128;
      for (int i = threadIdx.x - 320; i < nrows * lines; i += 64) {
        const char* g = reinterpret_cast<const char*>(p.gate + static_cast<size_t>(q0 + i / lines) * p.ld_gate + h * p.vdim) + (i % lines) * 128;
        asm volatile("prefetch.global.L2 [%0];" ::"l"(g));
      }
    } else if (warp == WARPS + 1) {
      if (lane == 0) {
        const uint32_t aQ = smem_u32(sQ), aK = smem_u32(sK), aV = smem_u32(sV);
        const uint32_t idesc_o = make_idesc_bf16(LA_BM, (p.vdim + 15) & ~15, 0, 1);
        const int steps_n = (p.dim + 15) >> 4, steps_r = (p.rot + 15) >> 4;
        // descriptors advance by their 16-byte-unit offsets: 2 per 16 K-major columns, 128 per 16 MN-major key rows
        const uint64_t dq0 = make_smem_desc(aQ, 16, 1024), dk0 = make_smem_desc(aK, 16, 1024), dv0 = make_smem_desc(aV, KPANEL, 1024);
        auto issue_s = [&](int x, int ks) {   // S_x = Q_x K^T, keys in stage ks
          uint64_t qd = dq0 + ((x * q_bytes) >> 4), kd = dk0 + ((ks * k_bytes) >> 4);
          const uint32_t d = tmem_base + x * BN;
          if constexpr (SN > 0) {
#pragma unroll
            for (int t = 0; t < SN + SR; ++t) {
              const int c = t < SN ? (t >> 2) : (SN + 3) / 4 + ((t - SN) >> 2), w = 2 * ((t < SN ? t : t - SN) & 3);
              umma_bf16(d, qd + c * (LA_QPANEL >> 4) + w, kd + c * (KPANEL >> 4) + w, IDESC_S, t ? 1u : 0u);
            }
            umma_commit(&bars->s_full[x]);
            return;
          }
          uint32_t acc = 0u;
          for (int c = 0; c < kp; ++c) {
            const int left = c < pn ? steps_n - 4 * c : steps_r - 4 * (c - pn);
            umma_bf16(d, qd, kd, IDESC_S, acc);
            if (left > 1) umma_bf16(d, qd + 2, kd + 2, IDESC_S, 1u);
            if (left > 2) umma_bf16(d, qd + 4, kd + 4, IDESC_S, 1u);
            if (left > 3) umma_bf16(d, qd + 6, kd + 6, IDESC_S, 1u);
            acc = 1u;
            qd += LA_QPANEL >> 4;
            kd += KPANEL >> 4;
          }
          umma_commit(&bars->s_full[x]);
        };
        auto issue_pv = [&](int x, int vs, bool first) {   // O_x += P_x V (stage vs), P_x over the first half of (every part of) S_x
          const uint64_t vd = dv0 + ((vs * v_bytes) >> 4);
          const uint32_t d = tmem_base + O_COL + x * O_WIDTH, a = tmem_base + x * BN;
#pragma unroll
          for (int t = 0; t < BN / 16; ++t)
            umma_bf16_ts(d, a + t * 8 + (t * 16 / (BN / SPLIT)) * (BN / SPLIT / 2), vd + t * 128, idesc_o, (first && t == 0) ? 0u : 1u);
        };
        bool ok = mbar_wait(&bars->q_full[0], 0, abort_flag, p.err, ERR_WAIT_ATTN) &&
                  mbar_wait(&bars->k_full[0], 0, abort_flag, p.err, ERR_WAIT_ATTN);
        if (ok) {
          tc_fence_after();
          issue_s(0, 0);
          ok = mbar_wait(&bars->q_full[1], 0, abort_flag, p.err, ERR_WAIT_ATTN);
          tc_fence_after();
          if (ok && je1 > 0 && jb1 == 0) issue_s(1, 0);
          umma_commit(&bars->k_empty[0]);
        }
        RingPos k, v;                        // stages of key block j + 1 and value block j
        for (int j = 0; j < nmax && ok; ++j, v.next(p.vst)) {
          k.next(p.kst);
          if (!mbar_wait(&bars->v_full[v.s], v.ph, abort_flag, p.err, ERR_WAIT_ATTN)) { ok = false; break; }
          if (j + 1 < nmax && !mbar_wait(&bars->k_full[k.s], k.ph, abort_flag, p.err, ERR_WAIT_ATTN)) { ok = false; break; }
          tc_fence_after();
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const int jb = x ? jb1 : 0, je = x ? je1 : je0;
            if (j >= jb && j < je) {
              if (!mbar_wait(&bars->p_ready[x], (j - jb) & 1, abort_flag, p.err, ERR_WAIT_ATTN)) { ok = false; break; }
              tc_fence_after();
              issue_pv(x, v.s, j == jb);
              if (j + 1 == je) umma_commit(&bars->o_final[x]);
            }
            if (j + 1 >= jb && j + 1 < je) issue_s(x, k.s);
          }
          if (!ok) break;
          umma_commit(&bars->v_empty[v.s]);
          if (j + 1 < nmax) umma_commit(&bars->k_empty[k.s]);
        }
      }
    }
  } else {
    if constexpr (SPLIT == 1) asm volatile("setmaxnreg.inc.sync.aligned.u32 216;");
    const int x = warp / (4 * SPLIT), part = (warp >> 2) % SPLIT;   // tile, part of its columns
    const int quad = warp & 3;
    const int jb = x ? jb1 : 0, je = x ? je1 : je0;
    // blocks [j_lo, j_hi) are visible to every row of the tile; the others are masked
    const int lo_last = max(kbase, s0 + (x ? last_b : last_a) - p.window + 1);
    const int j_lo = nkb + (lo_last - kstart + BN - 1) / BN, j_hi = nkb + (s0 + x * LA_BM + 1 - kstart) / BN;
    const int hi = s0 - kstart + x * LA_BM + quad * 32 + lane;   // newest visible key of this thread's row, from kstart
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t ts = tmem_base + x * BN + lane_addr;
    const uint32_t to = tmem_base + O_COL + x * O_WIDTH + lane_addr;
    float scale_log2 = p.scale_log2;
    const float* btab = nullptr;
    if constexpr (KIND == BIAS) {
      if (p.temp_every > 0)
        scale_log2 *= 1.f + p.temp_coef * logf(static_cast<float>((kstart + hi - kbase + 1) / p.temp_every + 1));
      btab = p.bias + static_cast<size_t>(h) * p.ld_bias + LA_BIAS_LEAD;
    }
    float m = la_bounded(KIND) ? 0.f : -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = jb; j < je && ok; ++j) {
      if (!mbar_wait(&bars->s_full[x], (j - jb) & 1, abort_flag, p.err, ERR_WAIT_ATTN)) { ok = false; break; }
      tc_fence_after();
      if constexpr (la_bounded(KIND)) {       // 32 columns at a time: no maximum to wait for
        const bool edge = j < j_lo || j >= j_hi;
        const int off = block_key(j) - kstart, cmax = hi - off, cmin = max(kbase - kstart - off, cmax - p.window + 1);
        const int ckeep = la_keeps(KIND) ? kbase + p.keep - kstart - off : 0;            // columns in front of it are kept keys
        float2 rs = make_float2(0.f, 0.f);
        constexpr int COLS = BN / SPLIT;
#pragma unroll
        for (int c0 = 0; c0 < COLS; c0 += 32) {
          const int c = part * COLS + c0;
          uint32_t raw[32], packed[16];
          tmem_ld_32x32(ts + c, raw);
          tmem_ld_wait(raw);
          float sv[32];
#pragma unroll
          for (int i = 0; i < 32; ++i) sv[i] = __uint_as_float(raw[i]);
          float2 r2[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
          auto weigh = [&](auto cap, auto masked) {
            r2[0] = r2[1] = make_float2(0.f, 0.f);
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              float2 y = cap(i);
              if constexpr (decltype(masked)::value) {
                if ((c + i < cmin && (!la_keeps(KIND) || c + i >= ckeep)) || c + i > cmax) y.x = -INFINITY;
                if ((c + i + 1 < cmin && (!la_keeps(KIND) || c + i + 1 >= ckeep)) || c + i + 1 > cmax) y.y = -INFINITY;
              }
              const float2 pr = make_float2(ex2_approx(y.x), ex2_approx(y.y));
              r2[(i >> 1) & 1] = fadd2(r2[(i >> 1) & 1], pr);
              packed[i >> 1] = pack_bf16x2(pr.x, pr.y);
            }
          };
          auto small = [&](int i) { return cap_small(make_float2(sv[i], sv[i + 1]), p); };
          if constexpr (KIND == SMALL) {
            auto plain = [&](int i) { return fmul2(make_float2(sv[i], sv[i + 1]), make_float2(scale_log2, scale_log2)); };
            if (edge) weigh(plain, std::true_type());
            else weigh(plain, std::false_type());
          } else if (__all_sync(0xffffffffu, max_abs(sv) <= p.poly_max)) {
            if (edge) weigh(small, std::true_type());
            else weigh(small, std::false_type());
          } else {
            weigh([&](int i) { return make_float2(cap_any(sv[i], p), cap_any(sv[i + 1], p)); }, std::true_type());
          }
          rs = fadd2(rs, fadd2(r2[0], r2[1]));
          tmem_st_32x16(ts + part * (COLS / 2) + (c >> 1), packed);
        }
        l += rs.x + rs.y;
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&bars->p_ready[x]);
      } else {
        float sv[BN];
#pragma unroll
        for (int c = 0; c < BN; c += 32) {
          uint32_t v[32];
          tmem_ld_32x32(ts + c, v);
#pragma unroll
          for (int i = 0; i < 32; ++i) sv[c + i] = __uint_as_float(v[i]);
        }
        tmem_ld_wait();
        if constexpr (KIND == CAPPED || KIND == KEPT) {
          if (p.capped) {
          if (__all_sync(0xffffffffu, max_abs(sv) <= p.poly_max)) {
#pragma unroll
            for (int i = 0; i < BN; i += 2) {
              const float2 y = cap_small(make_float2(sv[i], sv[i + 1]), p);
              sv[i] = y.x;
              sv[i + 1] = y.y;
            }
          } else {
#pragma unroll
            for (int i = 0; i < BN; ++i) sv[i] = cap_any(sv[i], p);
          }
        }
        }
        if (j < j_lo || j >= j_hi) {
          const int off = block_key(j) - kstart, cmax = hi - off, cmin = max(kbase - kstart - off, cmax - p.window + 1);
          const int ckeep = la_keeps(KIND) ? kbase + p.keep - kstart - off : cmin;       // columns in front of it are kept keys
#pragma unroll
          for (int i = 0; i < BN; ++i)
            if ((i < cmin && (!la_keeps(KIND) || i >= ckeep)) || i > cmax) sv[i] = -INFINITY;
        }
        float mul = KIND >= CAPPED && p.capped ? 1.f : scale_log2, add = 0.f;      // log2 score = mul * sv + add
        if constexpr (KIND == BIAS) {
          const int d0 = s0 - kstart + x * LA_BM - j * BN, far = p.bias_len - 1;   // distance of the tile's first row to the block's first key
          const int dmin = d0 - (BN - 1), dmax = d0 + LA_BM - 1;
          if (dmin >= far || (dmin >= 0 && p.bucket[dmin] == p.bucket[min(dmax, far)])) {
            add = btab[min(dmin, far)];
          } else {
            const float* b = btab + (hi - j * BN);
#pragma unroll
            for (int i = 0; i < BN; ++i) sv[i] = fmaf(sv[i], scale_log2, b[-i]);
            mul = 1.f;
          }
        }
        float mx4[4] = {sv[0], sv[1], sv[2], sv[3]};
#pragma unroll
        for (int i = 4; i + 7 < BN; i += 8) {
          mx4[0] = fmax3(mx4[0], sv[i], sv[i + 1]);
          mx4[1] = fmax3(mx4[1], sv[i + 2], sv[i + 3]);
          mx4[2] = fmax3(mx4[2], sv[i + 4], sv[i + 5]);
          mx4[3] = fmax3(mx4[3], sv[i + 6], sv[i + 7]);
        }
        mx4[0] = fmax3(mx4[0], sv[BN - 4], sv[BN - 3]);
        mx4[1] = fmax3(mx4[1], sv[BN - 2], sv[BN - 1]);
        const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
        const float m_new = fmaxf(m, fmaf(mx, mul, add));
        // raise the reference max only when it moved by more than the threshold (decided per warp)
        const bool grow = (m_new - m > RESCALE_THRESHOLD) || (m == -INFINITY);
        if (__any_sync(0xffffffffu, grow)) {
          const float alpha = (m == -INFINITY) ? 0.f : ex2_approx(m - m_new);
          if (j > jb) {
#pragma unroll 1
            for (int c = 0; c < p.vdim; c += 32) {
              uint32_t v[32];
              tmem_ld_32x32(to + c, v);
              tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
              tmem_st_32x32(to + c, v);
            }
          }
          l *= alpha;
          m = m_new;
        }
        const float neg_m = (m == -INFINITY) ? 0.f : add - m;   // a row may see nothing of the tile's first blocks
        const float2 neg_m2 = make_float2(neg_m, neg_m), scale2 = make_float2(mul, mul);
        float2 rs[4] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
        for (int c = 0; c < BN; c += 32) {
          uint32_t packed[16];
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const float2 a = ffma2(make_float2(sv[c + i], sv[c + i + 1]), scale2, neg_m2);
            const float2 pr = make_float2(ex2_approx(a.x), ex2_approx(a.y));
            rs[(i >> 1) & 3] = fadd2(rs[(i >> 1) & 3], pr);
            packed[i >> 1] = pack_bf16x2(pr.x, pr.y);
          }
          tmem_st_32x16(ts + (c >> 1), packed);
        }
        {
          const float2 t = fadd2(fadd2(rs[0], rs[1]), fadd2(rs[2], rs[3]));
          l += t.x + t.y;
        }
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&bars->p_ready[x]);
      }
    }
    if constexpr (SPLIT == 2) {
      if (je > jb) {                          // the row's other half of the sum, through the tile's queries: its last scores are formed
        float* sums = reinterpret_cast<float*>(sQ + x * q_bytes) + quad * 32 + lane;
        sums[part * LA_BM] = l;
        named_barrier_sync(1 + x, 256);
        l += sums[(part ^ 1) * LA_BM];
      }
    }
    if (ok && je > jb) {
      const int r = x * LA_BM + quad * 32 + lane;              // query of this thread inside the CTA's 256
      const bool live = r < nrows;
      const size_t t = live ? static_cast<size_t>(q0) + r : 0;
      __nv_bfloat16* orow = p.out + t * p.ld_out + h * p.vdim;
      if constexpr (KIND != LATENT) {
        float g = 1.f, den = l;
        if constexpr (KIND == BIAS) g = p.gate_mult / (1.f + __expf(-bf2f(p.gate[t * p.ld_gate + h])));
        if constexpr (KIND >= CAPPED)
          if (p.sink) den += ex2_approx(fmaf(p.sink[h], 1.4426950408889634f, -m));
        if (mbar_wait(&bars->o_final[x], 0, abort_flag, p.err, ERR_WAIT_ATTN)) {
          tc_fence_after();
          const float f = (l > 0.f) ? g / den : 0.f;
#pragma unroll 1
          for (int c = 32 * part; c < p.vdim; c += 32 * SPLIT) {
            uint32_t v[32];
            tmem_ld_32x32(to + c, v);
            tmem_ld_wait();
            if (live) {
#pragma unroll
              for (int q = 0; q < 4; ++q) {
                if (c + 8 * q < p.vdim) {
                  uint32_t o[4];
#pragma unroll
                  for (int i = 0; i < 4; ++i)
                    o[i] = pack_bf16x2(__uint_as_float(v[8 * q + 2 * i]) * f, __uint_as_float(v[8 * q + 2 * i + 1]) * f);
                  *reinterpret_cast<uint4*>(orow + c + 8 * q) = make_uint4(o[0], o[1], o[2], o[3]);
                }
              }
            }
          }
        }
      } else {
        const __nv_bfloat16* grow_ = p.gate + t * p.ld_gate + h * p.vdim;
        uint4 gq[16];                                             // up to 128 gate values, requested before the last product ends
        auto load_gate = [&](int c0) {
  #pragma unroll
          for (int q = 0; q < 16; ++q)
            if (c0 + 8 * q < p.vdim) gq[q] = *reinterpret_cast<const uint4*>(grow_ + c0 + 8 * q);
        };
        load_gate(0);
        if (mbar_wait(&bars->o_final[x], 0, abort_flag, p.err, ERR_WAIT_ATTN)) {
          tc_fence_after();
          const float inv_l = (l > 0.f) ? 1.f / l : 0.f;
  #pragma unroll 1
          for (int c0 = 0; c0 < p.vdim; c0 += 128) {
            if (c0) load_gate(c0);
  #pragma unroll
            for (int b = 0; b < 4; ++b) {
              const int c = c0 + 32 * b;
              if (c >= p.vdim) break;
              uint32_t v[32];
              tmem_ld_32x32(to + c, v);
              tmem_ld_wait();
              if (live) {
  #pragma unroll
                for (int q = 0; q < 4; ++q) {
                  if (c + 8 * q < p.vdim) {
                    const uint4 g4 = gq[4 * b + q];
                    const uint32_t gw[4] = {g4.x, g4.y, g4.z, g4.w};
                    uint32_t o[4];
  #pragma unroll
                    for (int i = 0; i < 4; ++i) {
                      const float2 g = unpack_bf16x2(gw[i]);
                      o[i] = pack_bf16x2(__uint_as_float(v[8 * q + 2 * i]) * inv_l / (1.f + __expf(-g.x)),
                                         __uint_as_float(v[8 * q + 2 * i + 1]) * inv_l / (1.f + __expf(-g.y)));
                    }
                    *reinterpret_cast<uint4*>(orow + c + 8 * q) = make_uint4(o[0], o[1], o[2], o[3]);
                  }
                }
              }
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == WARPS + 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

typedef CUresult (*EncodeTiledFnL)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                   const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                   CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// bf16 tensor [(heads,) rows, cols] with row pitch `ld` and head pitch `head` (elements); box: `box_rows` rows x 64 columns of
// one head, 128-byte swizzle.  heads = 0: two-dimensional.
static int make_tmap_rows(CUtensorMap* out, const void* base, uint64_t cols, uint64_t heads, uint64_t rows, uint64_t head, uint64_t ld,
                          uint32_t box_rows) {
  static EncodeTiledFnL enc = nullptr;
  if (!enc) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess ||
        q != cudaDriverEntryPointSuccess)
      return -1;
    enc = reinterpret_cast<EncodeTiledFnL>(ptr);
  }
  if ((reinterpret_cast<uintptr_t>(base) & 15) || (ld & 7) || (heads && (head & 7))) return -2;
  const int rank = heads ? 3 : 2;
  cuuint64_t dims[3] = {cols, rows, heads};
  cuuint64_t strides[2] = {ld * 2, head * 2};
  cuuint32_t box[3] = {64, box_rows, 1};
  cuuint32_t estr[3] = {1, 1, 1};
  return enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void*>(base), dims, strides, box, estr,
             CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
             CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : -3;
}

struct LatentAttnPlan { int bn, kst, vst, smem; };

// Key-block width and ring depths for the given sizes; bn = 0: not covered.
static LatentAttnPlan latent_attn_plan(int dim, int rot, int vdim) {
  LatentAttnPlan none = {0, 0, 0, 0};
  if ((dim & 7) || (rot & 7) || (vdim & 7) || dim <= 0 || rot < 0 || vdim <= 0) return none;
  const int kp = (dim + 63) / 64 + (rot + 63) / 64, pv = (vdim + 63) / 64;
  constexpr int LIMIT = 227 * 1024, FIXED = 1024 + 1024;   // barriers, alignment
  for (int bn = 128; bn >= 64; bn -= 64) {
    if (((vdim + 31) & ~31) > (512 - 2 * bn) / 2) continue;
    // 128-key blocks are worth a single value stage: the per-block synchronisation is the larger cost
    constexpr int STAGES[4][2] = {{3, 3}, {2, 3}, {2, 2}, {2, 1}};
    for (const auto& st : STAGES) {
      const int need = 2 * kp * LA_QPANEL + (st[0] * kp + st[1] * pv) * bn * 128 + FIXED;
      if (need <= LIMIT) return {bn, st[0], st[1], need};
    }
  }
  return none;
}

template <int BN, int SN, int SR, int KIND = LATENT>
static int launch_latent_attn(const CUtensorMap* tm, const LatentAttnParams& p, const LatentAttnPlan& plan, int n_tiles, cudaStream_t st) {
  auto kern = latent_attn_kernel<BN, SN, SR, KIND>;
  static int configured = 0;
  if (configured < plan.smem) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, plan.smem) != cudaSuccess) return -10;
    configured = plan.smem;
  }
  kern<<<dim3(p.H, n_tiles), la_threads(KIND), plan.smem, st>>>(tm[0], tm[1], tm[2], tm[3], tm[4], p);
  return cudaGetLastError() == cudaSuccess ? 0 : -11;
}

static int dispatch_latent_attn(const CUtensorMap* tm, const LatentAttnParams& p, const LatentAttnPlan& plan, int n_tiles, cudaStream_t st) {
  const int sn = (p.dim + 15) / 16, sr = (p.rot + 15) / 16;
  if (plan.bn == 64) return launch_latent_attn<64, 0, 0>(tm, p, plan, n_tiles, st);
  if (sn == 8 && sr == 4) return launch_latent_attn<128, 8, 4>(tm, p, plan, n_tiles, st);   // 128 + 64
  if (sn == 8 && sr == 2) return launch_latent_attn<128, 8, 2>(tm, p, plan, n_tiles, st);   // 128 + 32
  if (sn == 6 && sr == 2) return launch_latent_attn<128, 6, 2>(tm, p, plan, n_tiles, st);   //  96 + 32
  if (sn == 4 && sr == 4) return launch_latent_attn<128, 4, 4>(tm, p, plan, n_tiles, st);   //  64 + 64
  if (sn == 4 && sr == 2) return launch_latent_attn<128, 4, 2>(tm, p, plan, n_tiles, st);   //  64 + 32
  return launch_latent_attn<128, 0, 0>(tm, p, plan, n_tiles, st);
}

template <int KIND>
static int dispatch_grouped(const CUtensorMap* tm, const LatentAttnParams& p, const LatentAttnPlan& plan, int n_tiles, cudaStream_t st) {
  if (plan.bn == 64) return launch_latent_attn<64, 0, 0, KIND>(tm, p, plan, n_tiles, st);
  switch ((p.dim + 15) / 16) {
    case 8: return launch_latent_attn<128, 8, 0, KIND>(tm, p, plan, n_tiles, st);
    case 6: return launch_latent_attn<128, 6, 0, KIND>(tm, p, plan, n_tiles, st);
    case 4: return launch_latent_attn<128, 4, 0, KIND>(tm, p, plan, n_tiles, st);
    default: return launch_latent_attn<128, 0, 0, KIND>(tm, p, plan, n_tiles, st);
  }
}

// tanh(t) = t (c0 + c1 t^2 + c2 t^4) on |t| <= 0.3 to 4e-7: interpolation of tanh(sqrt(u)) / sqrt(u) at Chebyshev nodes of [0, 0.09].
static constexpr double TANH_RANGE = 0.3, TANH_POLY[3] = {0.9999988351, -0.3330998880, 0.1263358239};

}  // namespace b200

using namespace b200;

B200_API int b200_latent_attention_supported(int dim, int rot, int vdim) { return rot > 0 && latent_attn_plan(dim, rot, vdim).bn > 0; }

// q: [T, ld_q] (head h at column h (dim + rot)), kn / v: [K, ld_kv] (head h at column h dim / h vdim), kr: [K, ld_kr],
// gate: [T, ld_gate], out: [T, ld_out]; tiles: int4 [n_tiles] as in LatentAttnParams.
B200_API int b200_latent_attention(const void* q, const void* kn, const void* kr, const void* v, const void* gate, void* out,
                                   const int* tiles, int n_tiles, int T, int K, int H, int dim, int rot, int vdim, int ld_q, int ld_kv,
                                   int ld_kr, int ld_gate, int ld_out, int window, float scale, void* stream, int* err) {
  const LatentAttnPlan plan = latent_attn_plan(dim, rot, vdim);
  if (!plan.bn || rot <= 0 || n_tiles <= 0 || n_tiles > 65535 || H <= 0 || T <= 0 || K <= 0 || window <= 0) return -1;
  if ((reinterpret_cast<uintptr_t>(gate) & 15) || (reinterpret_cast<uintptr_t>(out) & 15) || (ld_gate & 7) || (ld_out & 7)) return -2;
  CUtensorMap tm[5];
  const __nv_bfloat16* qb = reinterpret_cast<const __nv_bfloat16*>(q);
  int rc = make_tmap_rows(&tm[0], qb, dim, H, T, dim + rot, ld_q, LA_BM);
  if (!rc) rc = make_tmap_rows(&tm[1], qb + dim, rot, H, T, dim + rot, ld_q, LA_BM);
  if (!rc) rc = make_tmap_rows(&tm[2], kn, dim, H, K, dim, ld_kv, plan.bn);
  if (!rc) rc = make_tmap_rows(&tm[3], kr, rot, 0, K, 0, ld_kr, plan.bn);
  if (!rc) rc = make_tmap_rows(&tm[4], v, vdim, H, K, vdim, ld_kv, plan.bn);
  if (rc) return rc;
  LatentAttnParams p = {};
  p.H = H; p.dim = dim; p.rot = rot; p.vdim = vdim; p.window = window;
  p.pn = (dim + 63) / 64; p.pr = (rot + 63) / 64; p.pv = (vdim + 63) / 64;
  p.kst = plan.kst; p.vst = plan.vst;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.tiles = reinterpret_cast<const int4*>(tiles);
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate); p.ld_gate = ld_gate;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ld_out = ld_out;
  p.err = err;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return dispatch_latent_attn(tm, p, plan, n_tiles, st);
}

B200_API int b200_biased_attention_supported(int dim, int vdim) { return latent_attn_plan(dim, 0, vdim).bn > 0; }
B200_API int b200_biased_attention_pad(int tail) { return tail ? LA_BIAS_TAIL : LA_BIAS_LEAD; }

// q: [T, ld_q] (head h at column h dim), k / v: cache [K, ld_kv] (head g at column g dim / g vdim), gate: [T, ld_gate] (head h at
// column h), out: [T, ld_out]; tiles as in LatentAttnParams; bias, bucket: see there.  scale > 0, temp_coef >= 0.
B200_API int b200_biased_attention(const void* q, const void* k, const void* v, const void* gate, void* out, const int* tiles,
                                   const float* bias, const int* bucket, int n_tiles, int T, int K, int H, int G, int dim, int vdim,
                                   int ld_q, int ld_kv, int ld_gate, int ld_out, int bias_len, int ld_bias, int temp_every,
                                   float temp_coef, float scale, float gate_mult, void* stream, int* err) {
  const LatentAttnPlan plan = latent_attn_plan(dim, 0, vdim);
  if (!plan.bn || n_tiles <= 0 || n_tiles > 65535 || H <= 0 || G <= 0 || H % G || T <= 0 || K <= 0 || bias_len <= 0 || !(scale > 0.f) ||
      temp_coef < 0.f || ld_bias < LA_BIAS_LEAD + bias_len + LA_BIAS_TAIL) return -1;
  if ((reinterpret_cast<uintptr_t>(out) & 15) || (ld_out & 7)) return -2;
  CUtensorMap tm[5];
  int rc = make_tmap_rows(&tm[0], q, dim, H, T, dim, ld_q, LA_BM);
  if (!rc) rc = make_tmap_rows(&tm[2], k, dim, G, K, dim, ld_kv, plan.bn);
  if (!rc) rc = make_tmap_rows(&tm[4], v, vdim, G, K, vdim, ld_kv, plan.bn);
  if (rc) return rc;
  tm[1] = tm[0];
  tm[3] = tm[2];
  LatentAttnParams p = {};
  p.H = H; p.dim = dim; p.rot = 0; p.vdim = vdim; p.window = 1 << 30;
  p.pn = (dim + 63) / 64; p.pr = 0; p.pv = (vdim + 63) / 64;
  p.kst = plan.kst; p.vst = plan.vst;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.tiles = reinterpret_cast<const int4*>(tiles);
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate); p.ld_gate = ld_gate;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ld_out = ld_out;
  p.err = err;
  p.group = H / G; p.bias = bias; p.bucket = bucket; p.bias_len = bias_len; p.ld_bias = ld_bias;
  p.temp_every = temp_every; p.temp_coef = temp_coef; p.gate_mult = gate_mult;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return dispatch_grouped<BIAS>(tm, p, plan, n_tiles, st);
}

B200_API int b200_capped_attention_supported(int dim, int vdim) { return latent_attn_plan(dim, 0, vdim).bn > 0; }

// q: [T, ld_q] (head h at column h dim), k / v: key stream [K, ld_kv] (head g at column g dim / g vdim), out: [T, ld_out]; tiles as in
// LatentAttnParams, none of them across the border of a chunk (whose first key is the tile's).  window: visible keys.  scale > 0;
// softcap 0: scores are not capped; sink: [H] or null.  keep: first keys of a sequence that stay visible; bound: no score is larger (0: not
// known).
B200_API int b200_capped_attention(const void* q, const void* k, const void* v, void* out, const int* tiles, const float* sink, int n_tiles, int T,
                                   int K, int H, int G, int dim, int vdim, int ld_q, int ld_kv, int ld_out, int window, int keep,
                                   float scale, float softcap, float bound, void* stream, int* err) {
  const LatentAttnPlan plan = latent_attn_plan(dim, 0, vdim);
  if (!plan.bn || n_tiles <= 0 || n_tiles > 65535 || H <= 0 || G <= 0 || H % G || T <= 0 || K <= 0 || window <= 0 || !(scale > 0.f) || softcap < 0.f || keep < 0) return -1;
  if ((reinterpret_cast<uintptr_t>(out) & 15) || (ld_out & 7)) return -2;
  CUtensorMap tm[5];
  int rc = make_tmap_rows(&tm[0], q, dim, H, T, dim, ld_q, LA_BM);
  if (!rc) rc = make_tmap_rows(&tm[2], k, dim, G, K, dim, ld_kv, plan.bn);
  if (!rc) rc = make_tmap_rows(&tm[4], v, vdim, G, K, vdim, ld_kv, plan.bn);
  if (rc) return rc;
  tm[1] = tm[0];
  tm[3] = tm[2];
  LatentAttnParams p = {};
  p.H = H; p.dim = dim; p.rot = 0; p.vdim = vdim; p.window = window;
  p.pn = (dim + 63) / 64; p.pr = 0; p.pv = (vdim + 63) / 64;
  p.kst = plan.kst; p.vst = plan.vst;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.tiles = reinterpret_cast<const int4*>(tiles);
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ld_out = ld_out;
  p.err = err;
  p.group = H / G; p.sink = sink;
  p.keep = keep;
  const bool small = softcap <= 0.f && bound > 0.f && bound * 1.4426950408889634f <= 80.f;
  bool bounded = false;
  if (softcap > 0.f) {
    const double x = static_cast<double>(scale) / softcap, cap = softcap * 1.4426950408889634;
    p.capped = 1;
    bounded = cap <= 80.0;              // weights lie in 2^(-80 .. 80): sums and products stay far inside fp32
    p.cap_log2 = static_cast<float>(cap);
    p.cap_exp = static_cast<float>(2.0 * x * 1.4426950408889634);
    double f = cap * x;                 // cap x^(2 i + 1)
    for (int i = 0; i < 3; ++i, f *= x * x) p.cap_poly[i] = static_cast<float>(TANH_POLY[i] * f);
    p.poly_max = x > 1e-6 && x < 1e6 ? static_cast<float>(TANH_RANGE / x) : -1.f;   // coefficients inside the range of fp32
  }
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (small) return dispatch_grouped<SMALL>(tm, p, plan, n_tiles, st);
  if (keep > 0) return dispatch_grouped<KEPT>(tm, p, plan, n_tiles, st);
  return bounded ? dispatch_grouped<BOUNDED>(tm, p, plan, n_tiles, st) : dispatch_grouped<CAPPED>(tm, p, plan, n_tiles, st);
}
