// Decode attention of latent-attention layers on the 5th-generation tensor cores: one query token per sequence, all heads of
// a sequence against the same cached latent rows, keys in a ring of `cap` slots (position p in slot p % cap).
//
// The cached rows are the large operand, so they fill the 128-row MMA dimension in both products:
//   S^T [128 keys, N heads] = rows [128 keys, ld] q^T           (K-major A; q already carried through the key up-projection)
//   O^T [128 latents, N heads] += rows^T [latents, 128 keys] P  (the same bytes as an MN-major A; P written by the softmax warps)
// One CTA per (key split, group of N heads, sequence).  A 128-key tile streams through a ring of 32 KB units (128 keys x 128
// columns) twice, once per product; the second pass hits L2.  S of tile i + 1 is issued before O of tile i, so loads and
// both products overlap the softmax.
//   warps 0-3  softmax: one key per thread, heads in groups of 16 that are read from tensor memory once for the maxima and
//              once for the weights (column reductions over the 128 keys by halving exchanges and shared memory), lazy
//              rescale of O^T, bf16 weights to shared memory (K-major, swizzled)
//   warp 4     TMA           warp 5  MMA issuer
// Every CTA leaves its unnormalised fp32 partial O [rank] per head with (max, sum); latent_expand merges the splits.
#include <cuda.h>

#include "common.cuh"

namespace b200 {

constexpr int LD_UNIT = 2 * 128 * 128;   // bytes of one ring unit: two 64-column panels of 128 keys
constexpr int LD_MAX_UNITS = 6;
constexpr int LD_RANK_CHUNKS = 7;

struct LatentDecodeParams {
  int H, rank, ld, window, cap, splits;
  int ring;                     // ring units
  float scale_log2;
  const int* pos;               // [B]
  const int* row;               // [B]
  float* part_o;                // [B, H, splits, rank padded to eight]
  float* part_ml;               // [B, H, splits, 2]
  int* err;
};

struct LatentDecodeBars {
  uint64_t q_full, full[LD_MAX_UNITS], empty[LD_MAX_UNITS], s_full[2], p_ready, o_done;
  uint32_t tmem_slot;
  int abort_flag;
};

// max (or sum) over the lanes of a warp of 16 values per lane by halving exchanges: lane l ends with value l % 16
template <bool SUM>
__device__ __forceinline__ float lane_reduce16(float (&v)[16]) {
  const int lane = threadIdx.x & 31;
  auto op = [](float a, float b) { return SUM ? a + b : fmaxf(a, b); };
#pragma unroll
  for (int off = 8; off > 0; off >>= 1) {
#pragma unroll
    for (int k = 0; k < off; ++k) {
      const bool up = lane & off;
      const float send = up ? v[k] : v[k + off], keep = up ? v[k + off] : v[k];
      v[k] = op(keep, __shfl_xor_sync(0xffffffffu, send, off));
    }
  }
  return op(v[0], __shfl_xor_sync(0xffffffffu, v[0], 16));
}

template <int N>
__global__ void __launch_bounds__(192, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmQ, const LatentDecodeParams p) {
  constexpr int QPANEL = N * 128;
  constexpr uint32_t IDESC_S = make_idesc_bf16(128, N, 0, 0);
  constexpr uint32_t IDESC_O = make_idesc_bf16(128, N, 1, 0);
  constexpr int TMEM_COLS = 512;

  pdl_trigger();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int panels = (p.ld + 63) >> 6;
  uint8_t* sR = smem;                            // ring
  uint8_t* sQ = sR + p.ring * LD_UNIT;
  uint8_t* sP = sQ + panels * QPANEL;            // [2 panels of 64 keys][N rows][128 bytes]
  float* s_wred = reinterpret_cast<float*>(sP + 2 * QPANEL);   // [4][N]
  float* s_sum = s_wred + 4 * N;                 // [4][N] running sums of every warp's keys
  float* s_m = s_sum + 4 * N;                    // [N] running reference maxima (log2 units)
  float* s_alpha = s_m + N;                      // [N]
  int* s_flag = reinterpret_cast<int*>(s_alpha + N);           // [2]
  LatentDecodeBars* bars = reinterpret_cast<LatentDecodeBars*>(s_flag + 4);
  volatile int* abort_flag = &bars->abort_flag;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, g = blockIdx.y, b = blockIdx.z;

  if (threadIdx.x == 128) {
    mbar_init(&bars->q_full, 1);
    for (int i = 0; i < LD_MAX_UNITS; ++i) {
      mbar_init(&bars->full[i], 1);
      mbar_init(&bars->empty[i], 1);
    }
    mbar_init(&bars->s_full[0], 1);
    mbar_init(&bars->s_full[1], 1);
    mbar_init(&bars->p_ready, 4);
    mbar_init(&bars->o_done, 1);
    bars->abort_flag = 0;
    fence_barrier_init();
    fence_proxy_async_smem();
  }
  if (threadIdx.x < N) s_m[threadIdx.x] = -INFINITY;
  for (int i = threadIdx.x; i < 4 * N; i += 192) s_sum[i] = 0.f;
  if (threadIdx.x < 2) s_flag[threadIdx.x] = 0;
  if (warp == 5) {
    tmem_alloc(&bars->tmem_slot, TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = bars->tmem_slot;
  pdl_wait();

  // The visible positions p, p - 1, ... occupy a circular run of slots that ends at p % cap: tiles end, end - 1, ... (modulo
  // the ring), of which this CTA takes every `splits`-th.
  const int pos = p.pos[b], seen = min(p.window, pos + 1);
  const int head_slot = pos % p.cap, ring_tiles = p.cap >> 7, end_tile = head_slot >> 7;
  const int in_end = (head_slot & 127) + 1;
  const int n_all = min(ring_tiles, 1 + (seen > in_end ? (seen - in_end + 127) >> 7 : 0));
  const int n = split < n_all ? (n_all - split + p.splits - 1) / p.splits : 0;
  const int units_s = (p.ld + 127) >> 7, units_o = (p.rank + 127) >> 7;
  auto tile_of = [&](int i) { int t = end_tile - (split + i * p.splits); return t < 0 ? t + ring_tiles : t; };

  if (warp == 4) {
    if (lane == 0 && n > 0) {
      const int row0 = p.row[b] * p.cap;
      mbar_expect_tx(&bars->q_full, panels * QPANEL);
      for (int c = 0; c < panels; ++c) tma_load_2d(sQ + c * QPANEL, &tmQ, &bars->q_full, c * 64, b * p.H + g * N);
      uint32_t it = 0, ph = 0;
      int s = 0;                         // ring unit, parity of the pass over the ring
      bool ok = true;
      auto load_tile = [&](int i, int units) {
        const int y = row0 + tile_of(i) * 128;
        for (int u = 0; u < units && ok; ++u, ++it) {
          if (!mbar_wait(&bars->empty[s], ph ^ 1, abort_flag, p.err, ERR_WAIT_STAGE_EMPTY)) { ok = false; break; }
          const bool two = u * 128 + 64 < p.ld;
          mbar_expect_tx(&bars->full[s], two ? LD_UNIT : LD_UNIT / 2);
          tma_load_2d(sR + s * LD_UNIT, &tmC, &bars->full[s], u * 128, y);
          if (two) tma_load_2d(sR + s * LD_UNIT + LD_UNIT / 2, &tmC, &bars->full[s], u * 128 + 64, y);
          if (++s == p.ring) { s = 0; ph ^= 1; }
        }
      };
      load_tile(0, units_s);
      for (int i = 0; i < n && ok; ++i) {
        if (i + 1 < n) load_tile(i + 1, units_s);
        if (ok) load_tile(i, units_o);
      }
      // every issued load must land before the CTA exits
      unsigned long long t0 = globaltimer_ns();
      while (!mbar_try_wait(&bars->q_full, 0) && globaltimer_ns() - t0 < WAIT_LIMIT_NS) {}
      for (uint32_t j = it > static_cast<uint32_t>(p.ring) ? it - p.ring : 0; j < it; ++j) {
        t0 = globaltimer_ns();
        while (!mbar_try_wait(&bars->full[j % p.ring], (j / p.ring) & 1) && globaltimer_ns() - t0 < WAIT_LIMIT_NS) {}
      }
    }
  } else if (warp == 5) {
    if (lane == 0 && n > 0) {
      const uint64_t dA = make_smem_desc(smem_u32(sR), 16, 1024), dAt = make_smem_desc(smem_u32(sR), 128 * 128, 1024);
      const uint64_t dQ = make_smem_desc(smem_u32(sQ), 16, 1024), dP = make_smem_desc(smem_u32(sP), 16, 1024);
      int s = 0;
      uint32_t ph = 0;
      bool ok = mbar_wait(&bars->q_full, 0, abort_flag, p.err, ERR_WAIT_TMA_FULL);
      auto wait_unit = [&]() {
        if (!mbar_wait(&bars->full[s], ph, abort_flag, p.err, ERR_WAIT_TMA_FULL)) return false;
        tc_fence_after();
        return true;
      };
      auto free_unit = [&]() {
        umma_commit(&bars->empty[s]);
        if (++s == p.ring) { s = 0; ph ^= 1; }
      };
      auto issue_s = [&](int i) {          // S^T of the i-th tile into score buffer i & 1
        const uint32_t d = tmem_base + (i & 1) * N;
        for (int u = 0; u < units_s && ok; ++u) {
          if (!wait_unit()) { ok = false; break; }
          for (int c = 0; c < 2; ++c) {
            if (u * 2 + c >= panels) break;      // columns past ld are zero in both operands: whole panels are multiplied
            const uint64_t a = dA + ((s * LD_UNIT + c * (LD_UNIT / 2)) >> 4), q = dQ + (((u * 2 + c) * QPANEL) >> 4);
            umma_bf16(d, a, q, IDESC_S, (u | c) ? 1u : 0u);
            umma_bf16(d, a + 2, q + 2, IDESC_S, 1u);
            umma_bf16(d, a + 4, q + 4, IDESC_S, 1u);
            umma_bf16(d, a + 6, q + 6, IDESC_S, 1u);
          }
          free_unit();
        }
        if (ok) umma_commit(&bars->s_full[i & 1]);
      };
      if (ok) issue_s(0);
      for (int i = 0; i < n && ok; ++i) {
        if (i + 1 < n) issue_s(i + 1);     // its score buffer was read before P of tile i - 1 was published
        if (!ok || !mbar_wait(&bars->p_ready, i & 1, abort_flag, p.err, ERR_WAIT_ATTN)) break;
        tc_fence_after();
        for (int u = 0; u < units_o && ok; ++u) {
          if (!wait_unit()) { ok = false; break; }
          const uint64_t a = dAt + ((s * LD_UNIT) >> 4);
          const uint32_t d = tmem_base + (2 + u) * N;
#pragma unroll
          for (int t = 0; t < 8; ++t)      // 16 keys per step; keys 64.. lie in the second panel of P
            umma_bf16(d, a + t * 128, dP + (t >> 2) * (QPANEL >> 4) + (t & 3) * 2, IDESC_O, (i | t) ? 1u : 0u);
          free_unit();
        }
        if (ok) umma_commit(&bars->o_done);
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax: thread = key of the tile
    const int key = threadIdx.x;
    const uint32_t lane_addr = static_cast<uint32_t>(warp * 32) << 16;
    float* wred = s_wred + warp * N;
    float* wsum = s_sum + warp * N;
    // A wait that gave up (the abort flag then ends all others quickly) must not take threads away from the named barriers:
    // the loop runs on without waiting and nothing is stored.
    bool ok = true;
    for (int i = 0; i < n; ++i) {
      const int slot = tile_of(i) * 128 + key;
      int back = head_slot - slot;
      if (back < 0) back += p.cap;
      const float scale = back < seen ? p.scale_log2 : 0.f, shift = back < seen ? 0.f : -INFINITY;   // hidden key: -inf
      ok = ok && mbar_wait(&bars->s_full[i & 1], (i >> 1) & 1, abort_flag, p.err, ERR_WAIT_ATTN);
      __syncwarp();
      tc_fence_after();
      const uint32_t ts = tmem_base + (i & 1) * N + lane_addr;
#pragma unroll 1
      for (int c = 0; c < N; c += 16) {
        uint32_t v[16];
        float t[16];
        tmem_ld_32x16(ts + c, v);
        tmem_ld_wait();
#pragma unroll
        for (int k = 0; k < 16; ++k) t[k] = fmaf(__uint_as_float(v[k]), scale, shift);
        const float m = lane_reduce16<false>(t);
        if (lane < 16) wred[c + lane] = m;
      }
      named_barrier_sync(1, 128);
      if (key < N) {
        const float m_old = s_m[key];
        const float m_tile = fmaxf(fmaxf(s_wred[key], s_wred[N + key]), fmaxf(s_wred[2 * N + key], s_wred[3 * N + key]));
        const bool grow = m_tile > m_old + 8.f;           // also from -inf
        s_alpha[key] = grow ? (m_old == -INFINITY ? 0.f : exp2f(m_old - m_tile)) : 1.f;
        if (grow) {
          s_m[key] = m_tile;
          s_flag[i & 1] = 1;
        }
      }
      if (key == 0) s_flag[(i + 1) & 1] = 0;
      named_barrier_sync(1, 128);
      // P's buffer and O^T are free once the products of the previous tile are complete
      if (i > 0) ok = ok && mbar_wait(&bars->o_done, (i - 1) & 1, abort_flag, p.err, ERR_WAIT_ATTN);
      __syncwarp();
      tc_fence_after();
      if (i > 0 && s_flag[i & 1]) {
        for (int c = lane; c < N; c += 32) wsum[c] *= s_alpha[c];
        for (int u = 0; u < units_o; ++u) {
#pragma unroll 1
          for (int c = 0; c < N; c += 16) {
            uint32_t v[16];
            const uint32_t ta = tmem_base + (2 + u) * N + c + lane_addr;
            tmem_ld_32x16(ta, v);
            tmem_ld_wait();
#pragma unroll
            for (int k = 0; k < 16; ++k) v[k] = __float_as_uint(__uint_as_float(v[k]) * s_alpha[c + k]);
            tmem_st_32x16(ta, v);
          }
        }
        tmem_st_wait();
        __syncwarp();
      }
      uint8_t* prow = sP + (key >> 6) * QPANEL + (key & 7) * 2;
      const int chunk = (key & 63) >> 3;
#pragma unroll 1
      for (int c = 0; c < N; c += 16) {
        uint32_t v[16];
        float t[16];
        tmem_ld_32x16(ts + c, v);
        tmem_ld_wait();
#pragma unroll
        for (int k = 0; k < 16; k += 4) {
          const float4 m4 = *reinterpret_cast<const float4*>(s_m + c + k);   // finite: every tile has a visible key
          const float m[4] = {m4.x, m4.y, m4.z, m4.w};
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float e = exp2f(fmaf(__uint_as_float(v[k + j]), scale, shift) - m[j]);
            t[k + j] = e;
            *reinterpret_cast<__nv_bfloat16*>(prow + (c + k + j) * 128 + ((chunk ^ ((k + j) & 7)) << 4)) = f2bf(e);
          }
        }
        const float sum = lane_reduce16<true>(t);
        if (lane < 16) wsum[c + lane] += sum;
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->p_ready);
    }
    const int heads = min(N, p.H - g * N), ld_o = (p.rank + 7) & ~7;
    const size_t base = (static_cast<size_t>(b) * p.H + g * N) * p.splits + split;
    if (n > 0) {
      ok = ok && mbar_wait(&bars->o_done, (n - 1) & 1, abort_flag, p.err, ERR_WAIT_ATTN);
      __syncwarp();
      tc_fence_after();
#pragma unroll 1
      for (int u = 0; u < units_o; ++u) {
        const int r = u * 128 + warp * 32 + lane;
#pragma unroll 1
        for (int c = 0; c < N; c += 16) {
          uint32_t v[16];
          tmem_ld_32x16(tmem_base + (2 + u) * N + c + lane_addr, v);
          tmem_ld_wait();
          if (ok && r < p.rank) {
            float* dst = p.part_o + (base + static_cast<size_t>(c) * p.splits) * ld_o + r;
#pragma unroll
            for (int k = 0; k < 16; ++k)
              if (c + k < heads) dst[static_cast<size_t>(k) * p.splits * ld_o] = __uint_as_float(v[k]);
          }
        }
      }
    }
    named_barrier_sync(1, 128);
    if (ok && key < heads) {
      const size_t o = 2 * (base + static_cast<size_t>(key) * p.splits);
      p.part_ml[o] = s_m[key] * 0.6931471805599453f;      // -inf for an empty split
      p.part_ml[o + 1] = (s_sum[key] + s_sum[N + key]) + (s_sum[2 * N + key] + s_sum[3 * N + key]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
}

int make_tmap_2d_bf16(CUtensorMap* out, const void* base, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows,
                      uint32_t box_cols);

struct LatentDecodePlan { int n, ring, smem; };

// Head-group width and ring depth; n = 0: not covered by this kernel.
static LatentDecodePlan latent_decode_plan(int H, int rank, int ld) {
  constexpr int LIMIT = 227 * 1024;
  if (H <= 0 || rank <= 0 || ld < rank || (ld & 7)) return {0, 0, 0};
  const int chunks = (rank + 127) / 128, panels = (ld + 63) / 64;
  for (int n = H > 32 ? 64 : (H > 16 ? 32 : 16); n >= 16; n >>= 1) {
    if (chunks > LD_RANK_CHUNKS || (2 + chunks) * n > 512) continue;
    const int fixed = 1024 + (panels + 2) * n * 128 + 10 * n * 4 + 64 + 512;
    const int ring = (LIMIT - fixed) / LD_UNIT;
    if (ring >= 2) {
      const int r = ring < LD_MAX_UNITS ? ring : LD_MAX_UNITS;
      return {n, r, fixed + r * LD_UNIT};
    }
  }
  return {0, 0, 0};
}

template <int N>
static int launch_latent_decode(const CUtensorMap& tc, const CUtensorMap& tq, const LatentDecodeParams& p, int smem, int B, cudaStream_t st) {
  auto kern = latent_decode_kernel<N>;
  static int configured = 0;
  if (configured < smem) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -10;
    configured = smem;
  }
  if (launch_k(kern, dim3(p.splits, (p.H + N - 1) / N, B), dim3(192), static_cast<size_t>(smem), st, tc, tq, p) != cudaSuccess) return -11;
  return cudaGetLastError() == cudaSuccess ? 0 : -11;
}

}  // namespace b200

using namespace b200;

// heads per CTA, 0 if the sizes are not covered
B200_API int b200_latent_decode_group(int H, int rank, int ld) { return latent_decode_plan(H, rank, ld).n; }

// q: [B, H, ld] bf16; cache: [rows, cap, ld] bf16 (cap a multiple of 128); partials as in LatentDecodeParams.
B200_API int b200_latent_decode(const void* q, const void* cache, const int* pos, const int* row, float* part_o, float* part_ml, int B,
                                int H, int rank, int ld, int rows, int cap, int window, int splits, float scale, void* stream, int* err) {
  const LatentDecodePlan plan = latent_decode_plan(H, rank, ld);
  if (!plan.n || B <= 0 || B > 65535 || (cap & 127) || cap <= 0 || window <= 0 || window > cap || splits < 1 || splits > 32 || rows <= 0) return -1;
  CUtensorMap tc, tq;
  int rc = make_tmap_2d_bf16(&tc, cache, static_cast<uint64_t>(rows) * cap, ld, ld, 128, 64);
  if (!rc) rc = make_tmap_2d_bf16(&tq, q, static_cast<uint64_t>(B) * H, ld, ld, plan.n, 64);
  if (rc) return rc;
  LatentDecodeParams p = {};
  p.H = H; p.rank = rank; p.ld = ld; p.window = window; p.cap = cap; p.splits = splits; p.ring = plan.ring;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.pos = pos; p.row = row; p.part_o = part_o; p.part_ml = part_ml; p.err = err;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  switch (plan.n) {
    case 16: return launch_latent_decode<16>(tc, tq, p, plan.smem, B, st);
    case 32: return launch_latent_decode<32>(tc, tq, p, plan.smem, B, st);
    default: return launch_latent_decode<64>(tc, tq, p, plan.smem, B, st);
  }
}
