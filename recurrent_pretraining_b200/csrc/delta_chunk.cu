// Gated delta rule over packed prompts, in chunks of 128 tokens on the 5th-generation tensor cores.
//
// Inside a chunk, with F the running sum of log decays, k^ the unit keys and S the state in front of the chunk,
//   u_t = beta_t (v_t - exp(F_t) S^T k^_t - sum_(j < t) exp(F_t - F_j) (k^_t . k^_j) u_j),
// so that (I + A) U = diag(beta) (V - diag(exp F) K^ S) with A strictly lower triangular: with T = (I + A)^-1
//   U = U0 - W S,   U0 = T diag(beta) V,   W = T diag(beta exp F) K^
//   S' = exp(F_end) S + K^^T diag(exp(F_end - F)) U
//   o_t = exp(F_t) S^T q_t + sum_(j <= t) exp(F_t - F_j) (q_t . k^_j) u_j
//   delta_chunk : A, T, U0 and W                                per (chunk, head), in parallel
//   delta_state : U and the states in front of every chunk       per (sequence, head, value columns)
//   chunk_out   : o, head norm and output gate (memory_chunk.cu) per (chunk, head), in parallel
// T is formed by substitution (blocks of 16 rows, then pairs of blocks up to 128) in fp32, which stays accurate however alike the keys are.
// Keys enter the products as they are (bf16); what makes them unit vectors is a factor on the other operand.  T, W, U and S enter them as a
// bf16 head plus a bf16 remainder; decays, gates, sums and the carried state are fp32.
#include "memory_chunk.cuh"

namespace b200 {

int make_tmap_2d_bf16(CUtensorMap* out, const void* base, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows, uint32_t box_cols);
int make_tmap_2d_f32(CUtensorMap* out, const void* base, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows);

constexpr int DC_PITCH = 132;                  // floats per row of T in shared memory

struct DeltaChunkParams {
  int H, G, dim, vdim, vpad, pk, pv, ldv;      // vpad: value columns padded to 16; 64-column panels
  int ba_t, ba_h, ld_u;                        // strides of `ba` per token and per column; pitch of u
  const int4* chunks;                          // {first token, tokens, sequence, -}
  const int4* seqs;                            // {first chunk, chunks, cache row, first position}
  const float* ba;                             // [T, 2 H] (strided) projections of step size | decay
  const float *a_log, *dt_bias;                // [H]
  float* u0;                                   // [chunks * H, 128, vpad]
  __nv_bfloat16 *w_hi, *w_lo;                  // [chunks * H, 128, dim]
  float *prefix, *fk;                          // [chunks * H, 128]
  __nv_bfloat16* u;                            // [T, ld_u], head h at column h vdim
  __nv_bfloat16 *s_hi, *s_lo;                  // [chunks * H, vpad, dim]
  float* state;                                // cache [rows, H, dim, ldv]
  int* err;
};

struct DeltaBars {
  uint64_t k_full, v_full, s_done, w_done, u_done;
  uint32_t tmem_slot;
  int abort_flag;
  float red[16];
};

// T21 = -T22 A21 T11 for every pair of S x S blocks on the diagonal: TR x TC results per thread, 256 threads.  A21 T11 lies in the pair's
// block above the diagonal meanwhile, which is zero again afterwards (not after the last level).
template <int S, int TR, int TC>
__device__ __forceinline__ void join_blocks(float* M, int tid) {
  constexpr int COLS = S / TC, TILES = (S / TR) * COLS;
  static_assert(64 / S * TILES == 256, "one tile per thread");
  const int pair = tid / TILES, tile = tid % TILES, r = (tile / COLS) * TR, c = (tile % COLS) * TC;
  const int C0 = pair * 2 * S, R0 = C0 + S;
  float2 acc[TR][TC / 2];
  auto multiply = [&](const float* a, const float* b, int k0, int k1) {   // rows r.. of a times columns c.. of b
#pragma unroll
    for (int i = 0; i < TR; ++i)
#pragma unroll
      for (int j = 0; j < TC / 2; ++j) acc[i][j] = make_float2(0.f, 0.f);
    for (int k = k0; k < k1; k += 4) {
      float av[TR][4];
#pragma unroll
      for (int i = 0; i < TR; ++i) ld4(a + (r + i) * DC_PITCH + k, av[i]);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float2 bv[TC / 2];
        if constexpr (TC == 4) {
          const float4 t = *reinterpret_cast<const float4*>(b + (k + e) * DC_PITCH + c);
          bv[0] = make_float2(t.x, t.y);
          bv[1] = make_float2(t.z, t.w);
        } else {
          bv[0] = ld2(b + (k + e) * DC_PITCH + c);
        }
#pragma unroll
        for (int i = 0; i < TR; ++i)
#pragma unroll
          for (int j = 0; j < TC / 2; ++j) acc[i][j] = ffma2(make_float2(av[i][e], av[i][e]), bv[j], acc[i][j]);
      }
    }
  };
  auto put = [&](float* d, float f) {
#pragma unroll
    for (int i = 0; i < TR; ++i)
#pragma unroll
      for (int j = 0; j < TC / 2; ++j) st2(d + (r + i) * DC_PITCH + c + 2 * j, make_float2(f * acc[i][j].x, f * acc[i][j].y));
  };
  float* Y = M + C0 * DC_PITCH + R0;
  multiply(M + R0 * DC_PITCH + C0, M + C0 * DC_PITCH + C0, c & ~3, S);       // T11 is zero above its diagonal
  put(Y, 1.f);
  __syncthreads();
  multiply(M + R0 * DC_PITCH + R0, Y, 0, r + TR);                             // and so is T22
  put(M + R0 * DC_PITCH + C0, -1.f);
  __syncthreads();
  if (S < 64) {
    put(Y, 0.f);
    __syncthreads();
  }
}

// Thread: token t = thread & 127, its columns shared by the two halves of the CTA.  Tensor memory: key products, then T with W's column
// factors, then T with U0's (head and remainder, 64 columns each); products at 128.  Shared memory is used again so that two CTAs fit an SM:
// the values follow the keys, what leaves the CTA is staged over T.  KS: 16-column steps of the keys (0: read from the parameters).
template <int KS>
__global__ void __launch_bounds__(256, 2)
delta_chunk_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmWh,
                   const __grid_constant__ CUtensorMap tmWl, const __grid_constant__ CUtensorMap tmU, const DeltaChunkParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  DeltaBars* bars = reinterpret_cast<DeltaBars*>(smem);
  uint8_t* sK = smem + 1024;                   // keys, then values
  float* M = reinterpret_cast<float*>(sK + max(p.pk, p.pv) * MC_PANEL);   // [128][DC_PITCH]; later tiles of 16 KB for the copy engine
  uint8_t* stage = reinterpret_cast<uint8_t*>(M);
  float* sF = M + MC_C * DC_PITCH;             // [128] running sums (log2 units), step sizes, key factors, factors of W's columns
  float* sB = sF + MC_C;
  float* sR = sB + MC_C;
  float* sW = sR + MC_C;
  float* sP = sW + MC_C;                       // [2][128] partial sums
  volatile int* abort_flag = &bars->abort_flag;
  const int h = blockIdx.x, ch = blockIdx.y, tid = threadIdx.x, t = tid & 127, half = tid >> 7, warp = tid >> 5;
  const int4 c = p.chunks[ch];
  const int t0 = c.x, n = c.y;
  const size_t idx = static_cast<size_t>(ch) * p.H + h;
  if (tid == 0) {
    mbar_init(&bars->k_full, 1);
    mbar_init(&bars->v_full, 1);
    mbar_init(&bars->s_done, 1);
    mbar_init(&bars->w_done, 1);
    mbar_init(&bars->u_done, 1);
    bars->abort_flag = 0;
    fence_barrier_init();
    fence_proxy_async_smem();
    mbar_expect_tx(&bars->k_full, p.pk * MC_PANEL);
    for (int i = 0; i < p.pk; ++i) tma_load_3d(sK + i * MC_PANEL, &tmK, &bars->k_full, i * 64, t0, h / (p.H / p.G));
  }
  if (warp == 1) {
    tmem_alloc(&bars->tmem_slot, 256);
    tmem_relinquish();
  }
  float beta = 0.f, lg = 0.f;
  if (t < n) {
    const float* z = p.ba + static_cast<size_t>(t0 + t) * p.ba_t;
    beta = sigmoid_f(z[static_cast<size_t>(h) * p.ba_h]);
    lg = -expf(p.a_log[h]) * softplus_f(z[static_cast<size_t>(p.H + h) * p.ba_h] + p.dt_bias[h]);
  }
  const float F = chunk_prefix<false>(lg, bars->red);
  if (half == 0) {
    sF[t] = F * LOG2E;
    sB[t] = beta;
    p.prefix[idx * MC_C + t] = F;
  }
  tc_fence_before();
  __syncthreads();                             // barriers, tensor memory
  tc_fence_after();
  const uint32_t tmem = bars->tmem_slot;
  const uint32_t ta = tmem + (static_cast<uint32_t>((warp & 3) * 32) << 16);
  bool ok = mbar_wait(&bars->k_full, 0, abort_flag, p.err, ERR_WAIT_TMA_FULL);
  if (tid == 0 && ok) {
    tc_fence_after();
    const uint64_t dk = make_smem_desc(smem_u32(sK), 16, 1024);
    constexpr uint32_t idesc = make_idesc_bf16(128, MC_C, 0, 0);
    if constexpr (KS > 0) {
#pragma unroll
      for (int k = 0; k < KS; ++k) umma_bf16(tmem, dk + ((k >> 2) * (MC_PANEL >> 4) + 2 * (k & 3)), dk + ((k >> 2) * (MC_PANEL >> 4) + 2 * (k & 3)), idesc, k ? 1u : 0u);
    } else {
      for (int k = 0; k < (p.dim + 15) >> 4; ++k) umma_bf16(tmem, dk + ((k >> 2) * (MC_PANEL >> 4) + 2 * (k & 3)), dk + ((k >> 2) * (MC_PANEL >> 4) + 2 * (k & 3)), idesc, k ? 1u : 0u);
    }
    umma_commit(&bars->s_done);
  }
  float kk = 0.f;                              // this half's 64 columns of the row
  if (ok && half < p.pk) {
#pragma unroll 4
    for (int i = 0; i < 8; ++i) {
      float v[8];
      ld8(reinterpret_cast<const __nv_bfloat16*>(sK + half * MC_PANEL + t * 128 + ((i ^ (t & 7)) << 4)), v);
#pragma unroll
      for (int e = 0; e < 8; ++e) kk += v[e] * v[e];
    }
  }
  sP[half * MC_C + t] = kk;
  __syncthreads();
  const float rk = 1.f / sqrtf(sP[t] + sP[MC_C + t] + 1e-6f);
  if (half == 0) {
    sR[t] = rk;
    sW[t] = beta * rk * exp2f(sF[t]);
    p.fk[idx * MC_C + t] = rk;
  }
  __syncthreads();
  ok = ok && mbar_wait(&bars->s_done, 0, abort_flag, p.err, ERR_WAIT_TMEM_FULL);
  ok = __all_sync(0xffffffffu, ok);
  // A below the diagonal, zeros above
  const float arow = sF[t], brow = beta * rk;
  const int newest = (warp & 3) * 32 + 31;     // last row of this warp: nothing behind its column
  if (ok) tc_fence_after();
#pragma unroll 1
  for (int b = 0; b < 2; ++b) {
    const int c0 = 64 * half + 32 * b;
    float* m = M + t * DC_PITCH + c0;
    if (!ok || c0 > newest) {
#pragma unroll
      for (int i = 0; i < 32; i += 4) *reinterpret_cast<float4*>(m + i) = make_float4(0.f, 0.f, 0.f, 0.f);
    } else {
      uint32_t v[32];
      tmem_ld_32x32(ta + c0, v);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; i += 4) {
        float f[4], r[4], w[4];
        ld4(sF + c0 + i, f);
        ld4(sR + c0 + i, r);
#pragma unroll
        for (int e = 0; e < 4; ++e) w[e] = c0 + i + e < t ? __uint_as_float(v[i + e]) * brow * r[e] * ex2_approx(arow - f[e]) : 0.f;
        *reinterpret_cast<float4*>(m + i) = make_float4(w[0], w[1], w[2], w[3]);
      }
    }
  }
  __syncthreads();
  // T = (I + A)^-1: blocks of 16 rows by substitution, one column per thread
  if (tid < MC_C) {
    const int b0 = tid & ~15, col = tid & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float s = i == col ? 1.f : 0.f;
#pragma unroll
      for (int q = 0; q < (i + 3) / 4; ++q) {
        float a[4];
        ld4(M + (b0 + i) * DC_PITCH + b0 + 4 * q, a);
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (4 * q + e < i) s -= a[e] * x[4 * q + e];
      }
      x[i] = s;
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < 16; ++i) M[(b0 + i) * DC_PITCH + b0 + col] = x[i];
  }
  __syncthreads();
  join_blocks<16, 2, 2>(M, tid);
  join_blocks<32, 2, 4>(M, tid);
  join_blocks<64, 4, 4>(M, tid);
  // rows of T times column factors as head and remainder into tensor memory
  auto pack = [&](const float* factor) {
#pragma unroll 1
    for (int b = 0; b < 2; ++b) {
      const int c0 = 64 * half + 32 * b;
      uint32_t hi[16], lo[16];
      if (c0 > newest) {
#pragma unroll
        for (int i = 0; i < 16; ++i) hi[i] = lo[i] = 0u;
      } else {
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          float m[4], f[4];
          ld4(M + t * DC_PITCH + c0 + i, m);
          ld4(factor + c0 + i, f);
          split_pack(m[0] * f[0], m[1] * f[1], hi[i >> 1], lo[i >> 1]);
          split_pack(m[2] * f[2], m[3] * f[3], hi[(i >> 1) + 1], lo[(i >> 1) + 1]);
        }
      }
      tmem_st_32x16(ta + (c0 >> 1), hi);
      tmem_st_32x16(ta + 64 + (c0 >> 1), lo);
    }
    tmem_st_wait();
    tc_fence_before();
  };
  // T (tensor memory) times token rows of shared memory
  auto product = [&](uint64_t d, uint32_t idesc, uint64_t* bar) {
    tc_fence_after();
#pragma unroll
    for (int k = 0; k < 16; ++k) umma_bf16_ts(tmem + 128, tmem + k * 8, d + (k & 7) * 128, idesc, k ? 1u : 0u);
    umma_commit(bar);
  };
  pack(sW);
  __syncthreads();
  const uint64_t dkv = make_smem_desc(smem_u32(sK), MC_PANEL, 1024);
  if (tid == 0) {
    if (ok) product(dkv, make_idesc_bf16(128, (p.dim + 15) & ~15, 0, 1), &bars->w_done);
    else bars->abort_flag = 1;
  }
  ok = ok && mbar_wait(&bars->w_done, 0, abort_flag, p.err, ERR_WAIT_TMEM_FULL);
  ok = __all_sync(0xffffffffu, ok);
  if (ok) tc_fence_after();
  bool asked = false;                          // values on their way
  if (tid == 0 && ok) {                        // the keys have been read
    asked = true;
    mbar_expect_tx(&bars->v_full, p.pv * MC_PANEL);
    for (int i = 0; i < p.pv; ++i) tma_load_3d(sK + i * MC_PANEL, &tmV, &bars->v_full, i * 64, t0, h);
  }
  __syncwarp();
  pack(sB);
  __syncthreads();                             // T has left shared memory
  if (ok) {
    for (int c0 = 16 * half; c0 < 64 * p.pk; c0 += 32) {
      uint32_t r[16], hi[8], lo[8];
      tmem_ld_32x16(ta + 128 + c0, r);         // columns behind the last are not stored
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 8; ++i) split_pack(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1]), hi[i], lo[i]);
      uint8_t* d = stage + (c0 >> 6) * MC_PANEL + t * 128;
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        const int piece = (((c0 & 63) >> 3) + q) ^ (t & 7);
        *reinterpret_cast<uint4*>(d + (piece << 4)) = make_uint4(hi[4 * q], hi[4 * q + 1], hi[4 * q + 2], hi[4 * q + 3]);
        *reinterpret_cast<uint4*>(d + 2 * MC_PANEL + (piece << 4)) = make_uint4(lo[4 * q], lo[4 * q + 1], lo[4 * q + 2], lo[4 * q + 3]);
      }
    }
  }
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  if (tid == 0) {
    const bool vok = asked && mbar_wait(&bars->v_full, 0, abort_flag, p.err, ERR_WAIT_TMA_FULL);
    if (vok) {
      product(dkv, make_idesc_bf16(128, p.vpad, 0, 1), &bars->u_done);
      for (int i = 0; i < p.pk; ++i) {
        tma_store_2d(&tmWh, stage + i * MC_PANEL, i * 64, static_cast<int>(idx) * MC_C);
        tma_store_2d(&tmWl, stage + (2 + i) * MC_PANEL, i * 64, static_cast<int>(idx) * MC_C);
      }
      bulk_commit_group();
      bulk_wait_read_all();
    } else {
      bars->abort_flag = 1;
    }
  }
  __syncwarp();
  ok = ok && mbar_wait(&bars->u_done, 0, abort_flag, p.err, ERR_WAIT_TMEM_FULL);
  ok = __all_sync(0xffffffffu, ok);
  __syncthreads();                             // W's tiles have been read
  if (ok) {
    tc_fence_after();
    for (int v0 = 16 * half; v0 < p.vpad; v0 += 32) {
      uint32_t r[16];
      tmem_ld_32x16(ta + 128 + v0, r);
      tmem_ld_wait();
      uint8_t* d = stage + (v0 >> 5) * MC_PANEL + t * 128;                     // tiles of 32 fp32 columns
#pragma unroll
      for (int q = 0; q < 4; ++q)
        *reinterpret_cast<uint4*>(d + (((((v0 & 31) >> 2) + q) ^ (t & 7)) << 4)) = make_uint4(r[4 * q], r[4 * q + 1], r[4 * q + 2], r[4 * q + 3]);
    }
  }
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  if (tid == 0 && ok) {
    for (int i = 0; i < (p.vpad + 31) / 32; ++i) tma_store_2d(&tmU, stage + i * MC_PANEL, i * 32, static_cast<int>(idx) * MC_C);
    bulk_commit_group();
    bulk_wait_all();
  }
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, 256);
  }
}

// ------------------------------------------------------------------------------------------------ recurrence over chunks
struct DeltaStateBars {
  uint64_t w_full, k_full[2], u0_full;         // W (head, remainder), keys (every other chunk) and U0 of a chunk have landed
  uint64_t s_ready, x_done, u_ready, d_done;   // state in shared memory; W S formed; weighted U in shared memory; K^T U formed
  uint64_t s_free;                             // the state's tile has been copied out
  uint32_t tmem_slot;
  int abort_flag;
};

constexpr int DS_VC = 16;                      // value columns of a compute thread
__host__ __device__ constexpr int ds_threads(int vb) { return 128 * (vb / DS_VC) + 64; }
__host__ __device__ constexpr int ds_u0_tiles(int vb) { return (vb + 31) / 32; }

// CTA: VB value columns of one head of one sequence.  Compute warps: thread = token row of W S and key row of the state, sixteen columns; then a warp for the MMAs
// and one for the copies.  Heads and remainders of S (as rows) and of the weighted U (as columns) lie side by side: one product takes both.
template <int VB, int KS>
__global__ void __launch_bounds__(ds_threads(VB), 1)
delta_state_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmWh, const __grid_constant__ CUtensorMap tmWl,
                   const __grid_constant__ CUtensorMap tmU0, const __grid_constant__ CUtensorMap tmSh, const __grid_constant__ CUtensorMap tmSl,
                   const DeltaChunkParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int SPANEL = 2 * VB * 128, NG = VB / DS_VC, VC = DS_VC, U0T = ds_u0_tiles(VB), UPANELS = (2 * VB + 63) / 64, MMA_WARP = 4 * NG;
  DeltaStateBars* bars = reinterpret_cast<DeltaStateBars*>(smem);
  uint8_t* sWh = smem + 1024;
  uint8_t* sWl = sWh + p.pk * MC_PANEL;
  uint8_t* sK = sWl + p.pk * MC_PANEL;         // twice two panels: the product's 128 rows are key columns
  uint8_t* sU = sK + 4 * MC_PANEL;             // token rows: head columns, remainder columns
  uint8_t* sU0 = sU + UPANELS * MC_PANEL;      // fp32 tiles [128][32]
  uint8_t* sS = sU0 + U0T * MC_PANEL;           // value rows of the head, then of the remainder; key columns
  volatile int* abort_flag = &bars->abort_flag;
  const int v0 = blockIdx.x * VB, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int4 sq = p.seqs[blockIdx.z];
  const int c0 = sq.x, nc = sq.y, hk = h / (p.H / p.G);
  auto load_w = [&](int c) {
    const int row = ((c0 + c) * p.H + h) * MC_C;
    mbar_expect_tx(&bars->w_full, 2 * p.pk * MC_PANEL);
    for (int i = 0; i < p.pk; ++i) {
      tma_load_2d(sWh + i * MC_PANEL, &tmWh, &bars->w_full, i * 64, row);
      tma_load_2d(sWl + i * MC_PANEL, &tmWl, &bars->w_full, i * 64, row);
    }
  };
  auto load_u0 = [&](int c) {
    const int row = ((c0 + c) * p.H + h) * MC_C;
    mbar_expect_tx(&bars->u0_full, U0T * MC_PANEL);
    for (int i = 0; i < U0T; ++i) tma_load_2d(sU0 + i * MC_PANEL, &tmU0, &bars->u0_full, v0 + 32 * i, row);
  };
  auto load_k = [&](int t0, int b) {
    mbar_expect_tx(&bars->k_full[b], p.pk * MC_PANEL);
    for (int i = 0; i < p.pk; ++i) tma_load_3d(sK + (2 * b + i) * MC_PANEL, &tmK, &bars->k_full[b], i * 64, t0, hk);
  };
  if (tid == 32 * MMA_WARP + 32) {
    mbar_init(&bars->w_full, 1);
    mbar_init(&bars->k_full[0], 1);
    mbar_init(&bars->k_full[1], 1);
    mbar_init(&bars->u0_full, 1);
    mbar_init(&bars->s_ready, 4 * NG);
    mbar_init(&bars->x_done, 1);
    mbar_init(&bars->u_ready, 4 * NG);
    mbar_init(&bars->d_done, 1);
    mbar_init(&bars->s_free, 1);
    bars->abort_flag = 0;
    fence_barrier_init();
    fence_proxy_async_smem();
    load_w(0);
    load_u0(0);
    load_k(p.chunks[c0].x, 0);
    if (nc > 1) load_k(p.chunks[c0 + 1].x, 1);
  }
  if (warp == MMA_WARP) {
    tmem_alloc(&bars->tmem_slot, 4 * VB);
    tmem_relinquish();
  }
  for (int i = tid; i < p.pk * SPANEL / 16; i += ds_threads(VB)) reinterpret_cast<uint4*>(sS)[i] = make_uint4(0u, 0u, 0u, 0u);   // columns past dim stay zero
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_slot, tx = tmem, td = tmem + 2 * VB;
  auto wait = [&](uint64_t* bar, uint32_t ph, int code) { return mbar_wait(bar, ph, abort_flag, p.err, code); };
  if (warp == MMA_WARP) {
    if (lane == 0) {
      constexpr uint32_t idesc_x2 = make_idesc_bf16(128, 2 * VB, 0, 0), idesc_x = make_idesc_bf16(128, VB, 0, 0), idesc_d = make_idesc_bf16(128, 2 * VB, 1, 1);
      uint64_t dwh = make_smem_desc(smem_u32(sWh), 16, 1024), dwl = make_smem_desc(smem_u32(sWl), 16, 1024), ds = make_smem_desc(smem_u32(sS), 16, 1024),
                     dk = make_smem_desc(smem_u32(sK), MC_PANEL, 1024), du = make_smem_desc(smem_u32(sU), MC_PANEL, 1024);
      for (int c = 0; c < nc; ++c) {
        const uint32_t ph = c & 1;
        asm volatile("" : "+l"(dwh), "+l"(dwl), "+l"(ds), "+l"(dk), "+l"(du));      // descriptors are added up here, not kept for the whole loop
        if (!wait(&bars->w_full, ph, ERR_WAIT_TMA_FULL) || !wait(&bars->s_ready, ph, ERR_WAIT_TMEM_FULL)) break;
        tc_fence_after();
        if constexpr (KS > 0) {
#pragma unroll
          for (int k = 0; k < KS; ++k) {
            const int ao = (k >> 2) * (MC_PANEL >> 4) + 2 * (k & 3), so = (k >> 2) * (SPANEL >> 4) + 2 * (k & 3);
            umma_bf16(tx, dwh + ao, ds + so, idesc_x2, k ? 1u : 0u);
          }
#pragma unroll
          for (int k = 0; k < KS; ++k) {
            const int ao = (k >> 2) * (MC_PANEL >> 4) + 2 * (k & 3), so = (k >> 2) * (SPANEL >> 4) + 2 * (k & 3);
            umma_bf16(tx, dwl + ao, ds + so, idesc_x, 1u);
          }
        } else {
          for (int k = 0; k < (p.dim + 15) >> 4; ++k) {
            const int ao = (k >> 2) * (MC_PANEL >> 4) + 2 * (k & 3), so = (k >> 2) * (SPANEL >> 4) + 2 * (k & 3);
            umma_bf16(tx, dwh + ao, ds + so, idesc_x2, k ? 1u : 0u);
            umma_bf16(tx, dwl + ao, ds + so, idesc_x, 1u);
          }
        }
        umma_commit(&bars->x_done);
        if (!wait(&bars->k_full[ph], (c >> 1) & 1, ERR_WAIT_TMA_FULL) || !wait(&bars->u_ready, ph, ERR_WAIT_TMEM_FULL)) break;
        tc_fence_after();
        const uint64_t dkc = dk + ph * (2 * MC_PANEL >> 4);
#pragma unroll
        for (int k = 0; k < 8; ++k) umma_bf16(td, dkc + k * 128, du + k * 128, idesc_d, k ? 1u : 0u);
        umma_commit(&bars->d_done);
      }
    }
  } else if (warp == MMA_WARP + 1) {
    if (lane == 0) {
      int w = 1, u = 1, k = nc > 1 ? 2 : 1;              // loads issued
      bool ok = true;
      for (int c = 0; c < nc && ok; ++c) {
        const uint32_t ph = c & 1;
        const bool more = c + 1 < nc;
        const int next = c + 2 < nc ? p.chunks[c0 + c + 2].x : 0;
        ok = wait(&bars->s_ready, ph, ERR_WAIT_TMEM_FULL);
        if (!ok) break;
        const int row = ((c0 + c) * p.H + h) * p.vpad + v0;
        for (int i = 0; i < p.pk; ++i) {
          tma_store_2d(&tmSh, sS + i * SPANEL, i * 64, row);
          tma_store_2d(&tmSl, sS + i * SPANEL + VB * 128, i * 64, row);
        }
        bulk_commit_group();
        ok = wait(&bars->x_done, ph, ERR_WAIT_TMEM_FULL);
        if (ok && more) {
          load_w(c + 1);
          ++w;
        }
        bulk_wait_read_all();
        mbar_arrive(&bars->s_free);
        ok = ok && wait(&bars->u_ready, ph, ERR_WAIT_TMEM_FULL);
        if (ok && more) {
          load_u0(c + 1);
          ++u;
        }
        ok = ok && wait(&bars->d_done, ph, ERR_WAIT_TMEM_FULL);
        if (ok && c + 2 < nc) {
          load_k(next, ph);
          ++k;
        }
      }
      bulk_wait_all();
      const unsigned long long begin = globaltimer_ns();   // a copy in flight has to land before the CTA ends
      while (!(mbar_try_wait(&bars->w_full, (w - 1) & 1) && mbar_try_wait(&bars->u0_full, (u - 1) & 1) && mbar_try_wait(&bars->k_full[(k - 1) & 1], ((k - 1) >> 1) & 1) &&
               (k < 2 || mbar_try_wait(&bars->k_full[k & 1], ((k - 2) >> 1) & 1))) &&
             globaltimer_ns() - begin < WAIT_LIMIT_NS) {}
    }
  } else {
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const int r = tid & 127, vc = (tid >> 7) * VC;       // token of the chunk and key row of the state; first of this thread's columns
    float* st = p.state + ((static_cast<size_t>(sq.z) * p.H + h) * p.dim + r) * p.ldv + v0 + vc;
    float S[VC];
#pragma unroll
    for (int v = 0; v < VC; ++v) S[v] = sq.w != 0 && r < p.dim && v0 + vc + v < p.vdim ? st[v] : 0.f;
    auto put_state = [&]() {
      if (r < p.dim) {
        uint8_t* d = sS + (r >> 6) * SPANEL + vc * 128 + (r & 7) * 2;
        int piece = (r & 63) >> 3;
        asm volatile("" : "+r"(piece));                  // addresses are formed here, not kept for the whole loop
#pragma unroll
        for (int v = 0; v < VC; ++v) {
          const __nv_bfloat16 hi = f2bf(S[v]);
          const int off = v * 128 + ((piece ^ (v & 7)) << 4);
          *reinterpret_cast<__nv_bfloat16*>(d + off) = hi;
          *reinterpret_cast<__nv_bfloat16*>(d + VB * 128 + off) = f2bf(S[v] - bf2f(hi));
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->s_ready);
    };
    // v += f (head's columns + remainder's columns) of this thread's row
    auto add_columns = [&](uint32_t at, float f, float (&v)[16]) {
      uint32_t x[16];
      tmem_ld_32x16(at + lane_addr + vc, x);
      if constexpr (VB < 64) {
        uint32_t y[16];
        tmem_ld_32x16(at + lane_addr + VB + vc, y);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) v[i] += f * (__uint_as_float(x[i]) + __uint_as_float(y[i]));
      } else {                                           // one after the other: registers
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) v[i] += f * __uint_as_float(x[i]);
        tmem_ld_32x16(at + lane_addr + VB + vc, x);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) v[i] += f * __uint_as_float(x[i]);
      }
    };
    put_state();
    int4 ck;
    float F, Fend, fk;
    auto chunk_info = [&](int c) {
      const size_t at = (static_cast<size_t>(c0 + c) * p.H + h) * MC_C;
      ck = p.chunks[c0 + c];
      F = p.prefix[at + r];
      Fend = p.prefix[at + MC_C - 1];
      fk = p.fk[at + r];
    };
    chunk_info(0);
    for (int c = 0; c < nc; ++c) {
      const uint32_t ph = c & 1;
      const float f = r < ck.y ? expf(Fend - F) * fk : 0.f, a = expf(Fend);
      __nv_bfloat16* dst = r < ck.y ? p.u + static_cast<size_t>(ck.x + r) * p.ld_u + h * p.vdim + v0 : nullptr;
      bool ok = wait(&bars->u0_full, ph, ERR_WAIT_TMA_FULL) && wait(&bars->x_done, ph, ERR_WAIT_TMEM_FULL);
      if (!__all_sync(0xffffffffu, ok)) break;
      tc_fence_after();
      float u[16];
      int r7 = r & 7;
      asm volatile("" : "+r"(r7));
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        float z[4];
        ld4(reinterpret_cast<const float*>(sU0 + (vc >> 5) * MC_PANEL + r * 128 + (((((vc & 31) >> 2) + q) ^ r7) << 4)), z);
#pragma unroll
        for (int i = 0; i < 4; ++i) u[4 * q + i] = z[i];
      }
      add_columns(tx, -1.f, u);
#pragma unroll
      for (int q = 0; q < 2; ++q) {                      // pieces of eight values of the token's row
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) split_pack(u[8 * q + 2 * i] * f, u[8 * q + 2 * i + 1] * f, hi[i], lo[i]);
        const int ch = vc + 8 * q, cl = VB + ch;
        *reinterpret_cast<uint4*>(sU + (ch >> 6) * MC_PANEL + r * 128 + ((((ch & 63) >> 3) ^ r7) << 4)) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(sU + (cl >> 6) * MC_PANEL + r * 128 + ((((cl & 63) >> 3) ^ r7) << 4)) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->u_ready);
#pragma unroll
      for (int q = 0; q < 2; ++q)
        if (dst && v0 + vc + 8 * q < p.vdim)
          *reinterpret_cast<uint4*>(dst + vc + 8 * q) = make_uint4(pack_bf16x2(u[8 * q], u[8 * q + 1]), pack_bf16x2(u[8 * q + 2], u[8 * q + 3]),
                                                                   pack_bf16x2(u[8 * q + 4], u[8 * q + 5]), pack_bf16x2(u[8 * q + 6], u[8 * q + 7]));
      if (c + 1 < nc) chunk_info(c + 1);
      ok = wait(&bars->d_done, ph, ERR_WAIT_TMEM_FULL);
      if (!__all_sync(0xffffffffu, ok)) break;
      tc_fence_after();
#pragma unroll
      for (int i = 0; i < 16; ++i) S[i] *= a;
      add_columns(td, 1.f, S);
      if (c + 1 < nc) {
        ok = wait(&bars->s_free, ph, ERR_WAIT_TMEM_FULL);
        if (!__all_sync(0xffffffffu, ok)) break;
        put_state();
      } else if (r < p.dim) {
#pragma unroll
        for (int v = 0; v < VC; ++v)
          if (v0 + vc + v < p.vdim) st[v] = S[v];
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == MMA_WARP) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, 4 * VB);
  }
}

static int dc_smem_chunk(int pk, int pv) { return 1024 + 1024 + (pk > pv ? pk : pv) * MC_PANEL + (MC_C * DC_PITCH + 6 * MC_C) * 4; }
static int dc_smem_state(int pk, int vb) { return 1024 + 1024 + (2 * pk + 4 + (2 * vb + 63) / 64 + ds_u0_tiles(vb)) * MC_PANEL + pk * 2 * vb * 128; }

struct DeltaMaps { CUtensorMap k, v, wh, wl, u0, sh, sl; };

template <int KS>
static int launch_delta_chunk(const DeltaMaps& m, const DeltaChunkParams& p, int n_chunks, cudaStream_t st) {
  const int smem = dc_smem_chunk(p.pk, p.pv);
  if (cudaFuncSetAttribute(delta_chunk_kernel<KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
  delta_chunk_kernel<KS><<<dim3(p.H, n_chunks), 256, smem, st>>>(m.k, m.v, m.wh, m.wl, m.u0, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <int VB, int KS>
static int launch_delta_state(const DeltaMaps& m, const DeltaChunkParams& p, int n_seqs, cudaStream_t st) {
  const int smem = dc_smem_state(p.pk, VB);
  if (cudaFuncSetAttribute(delta_state_kernel<VB, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
  delta_state_kernel<VB, KS><<<dim3(p.vpad / VB, p.H, n_seqs), ds_threads(VB), smem, st>>>(m.k, m.wh, m.wl, m.u0, m.sh, m.sl, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <int VB>
static int dispatch_delta_state(const DeltaMaps& m, const DeltaChunkParams& p, int n_seqs, cudaStream_t st) {
  switch ((p.dim + 15) / 16) {
    case 8: return launch_delta_state<VB, 8>(m, p, n_seqs, st);
    case 6: return launch_delta_state<VB, 6>(m, p, n_seqs, st);
    case 4: return launch_delta_state<VB, 4>(m, p, n_seqs, st);
    default: return launch_delta_state<VB, 0>(m, p, n_seqs, st);
  }
}

}  // namespace b200

using namespace b200;

B200_API int b200_delta_chunk_supported(int dim, int vdim) {
  return dim > 0 && vdim > 0 && !(dim & 7) && !(vdim & 7) && dim <= 128 && vdim <= 128;
}

// k, v: columns of the activated rows [T, ld] (key head g at column g dim, head h at column h vdim).  parts: 1 single chunks, 2 recurrence.
B200_API int b200_delta_chunks(const void* k, const void* v, int ld, const DeltaChunkParams* Pp, int T, int n_chunks, int n_seqs, int parts, void* stream,
                               int* err) {
  DeltaChunkParams p = *Pp;
  if (!b200_delta_chunk_supported(p.dim, p.vdim) || T <= 0 || n_chunks <= 0 || n_chunks > 65535 || n_seqs <= 0 || n_seqs > 65535 || p.H <= 0 || p.H > 65535 ||
      p.G <= 0 || p.H % p.G || (ld & 7) || (p.ld_u & 7) || p.ldv < p.vdim || !p.ba || !p.a_log || !p.dt_bias || !p.state) return -1;
  if ((reinterpret_cast<uintptr_t>(p.u0) | reinterpret_cast<uintptr_t>(p.w_hi) | reinterpret_cast<uintptr_t>(p.w_lo) | reinterpret_cast<uintptr_t>(p.u)) & 15) return -1;
  p.vpad = (p.vdim + 15) & ~15;
  p.pk = (p.dim + 63) / 64;
  p.pv = (p.vdim + 63) / 64;
  p.err = err;
  // value columns per CTA of the recurrence: narrow while the machine has room for all CTAs at once
  const int vb = p.vpad % 32 ? 16 : p.vpad % 64 == 0 && static_cast<long long>(n_seqs) * p.H * (p.vpad / 32) > 148 ? 64 : 32;
  const uint64_t planes = static_cast<uint64_t>(n_chunks) * p.H;
  if (planes * MC_C > 0x7fffffffull) return -1;
  DeltaMaps m;
  int rc = make_tmap_planes(&m.k, k, p.dim, T, p.G, ld, p.dim, MC_C);
  if (!rc) rc = make_tmap_planes(&m.v, v, p.vdim, T, p.H, ld, p.vdim, MC_C);
  if (!rc) rc = make_tmap_2d_bf16(&m.wh, p.w_hi, planes * MC_C, p.dim, p.dim, MC_C, 64);
  if (!rc) rc = make_tmap_2d_bf16(&m.wl, p.w_lo, planes * MC_C, p.dim, p.dim, MC_C, 64);
  if (!rc) rc = make_tmap_2d_f32(&m.u0, p.u0, planes * MC_C, p.vpad, p.vpad, MC_C);
  if (!rc) rc = make_tmap_2d_bf16(&m.sh, p.s_hi, planes * p.vpad, p.dim, p.dim, vb, 64);
  if (!rc) rc = make_tmap_2d_bf16(&m.sl, p.s_lo, planes * p.vpad, p.dim, p.dim, vb, 64);
  if (rc) return rc;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (parts & 1) {
    switch ((p.dim + 15) / 16) {
      case 8: rc = launch_delta_chunk<8>(m, p, n_chunks, st); break;
      case 6: rc = launch_delta_chunk<6>(m, p, n_chunks, st); break;
      case 4: rc = launch_delta_chunk<4>(m, p, n_chunks, st); break;
      default: rc = launch_delta_chunk<0>(m, p, n_chunks, st);
    }
    if (rc) return rc;
  }
  if (parts & 2) return vb == 64 ? dispatch_delta_state<64>(m, p, n_seqs, st) : vb == 32 ? dispatch_delta_state<32>(m, p, n_seqs, st) : dispatch_delta_state<16>(m, p, n_seqs, st);
  return 0;
}
