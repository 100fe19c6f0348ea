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

constexpr int DC_PITCH = 132;                  // floats per row of T in shared memory
constexpr int DC_YPITCH = 68;

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
  uint64_t k_full, v_full, s_done, uw_done;
  uint32_t tmem_slot;
  int abort_flag;
  float red[16];
};

// T21 = -T22 A21 T11 for every pair of S x S blocks on the diagonal: TR x TC results per thread, 256 threads.
template <int S, int TR, int TC>
__device__ __forceinline__ void join_blocks(float* M, float* Y, int tid) {
  constexpr int COLS = S / TC, TILES = (S / TR) * COLS;
  static_assert(64 / S * TILES == 256, "one tile per thread");
  const int pair = tid / TILES, tile = tid % TILES, r = (tile / COLS) * TR, c = (tile % COLS) * TC;
  const int C0 = pair * 2 * S, R0 = C0 + S;
  float* y = Y + pair * S * (S + 4);
  float acc[TR][TC];
  auto multiply = [&](const float* a, int pa, const float* b, int pb, int k0, int k1) {   // rows r.. of a times columns c.. of b
#pragma unroll
    for (int i = 0; i < TR; ++i)
#pragma unroll
      for (int j = 0; j < TC; ++j) acc[i][j] = 0.f;
    for (int k = k0; k < k1; k += 4) {
      float av[TR][4];
#pragma unroll
      for (int i = 0; i < TR; ++i) ld4(a + (r + i) * pa + k, av[i]);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float bv[TC];
        if constexpr (TC == 4) {
          ld4(b + (k + e) * pb + c, bv);
        } else {
          const float2 t = ld2(b + (k + e) * pb + c);
          bv[0] = t.x;
          bv[1] = t.y;
        }
#pragma unroll
        for (int i = 0; i < TR; ++i)
#pragma unroll
          for (int j = 0; j < TC; ++j) acc[i][j] += av[i][e] * bv[j];
      }
    }
  };
  multiply(M + R0 * DC_PITCH + C0, DC_PITCH, M + C0 * DC_PITCH + C0, DC_PITCH, c & ~3, S);       // T11 is zero above its diagonal
#pragma unroll
  for (int i = 0; i < TR; ++i)
#pragma unroll
    for (int j = 0; j < TC; ++j) y[(r + i) * (S + 4) + c + j] = acc[i][j];
  __syncthreads();
  multiply(M + R0 * DC_PITCH + R0, DC_PITCH, y, S + 4, 0, r + TR);                               // and so is T22
#pragma unroll
  for (int i = 0; i < TR; ++i)
#pragma unroll
    for (int j = 0; j < TC; ++j) M[(R0 + r + i) * DC_PITCH + C0 + c + j] = -acc[i][j];
  __syncthreads();
}

// Thread: token t = thread & 127, its columns shared by the two halves of the CTA.  Tensor memory: key products, then beta-weighted T (head,
// remainder) over them; W's T at 128; U0 at 256; W at 384.
__global__ void __launch_bounds__(256, 1)
delta_chunk_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const DeltaChunkParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  DeltaBars* bars = reinterpret_cast<DeltaBars*>(smem);
  uint8_t* sK = smem + 1024;
  uint8_t* sV = sK + p.pk * MC_PANEL;
  float* M = reinterpret_cast<float*>(sV + p.pv * MC_PANEL);   // [128][DC_PITCH]
  float* Y = M + MC_C * DC_PITCH;                              // [64][DC_YPITCH]
  float* sF = Y + 64 * DC_YPITCH;                              // [128] running sums (log2 units), step sizes, key factors, partial sums [2][128]
  float* sB = sF + MC_C;
  float* sR = sB + MC_C;
  float* sP = sR + MC_C;
  volatile int* abort_flag = &bars->abort_flag;
  const int h = blockIdx.x, ch = blockIdx.y, tid = threadIdx.x, t = tid & 127, half = tid >> 7, warp = tid >> 5;
  const int4 c = p.chunks[ch];
  const int t0 = c.x, n = c.y;
  const size_t idx = static_cast<size_t>(ch) * p.H + h;
  if (tid == 0) {
    mbar_init(&bars->k_full, 1);
    mbar_init(&bars->v_full, 1);
    mbar_init(&bars->s_done, 1);
    mbar_init(&bars->uw_done, 1);
    bars->abort_flag = 0;
    fence_barrier_init();
    fence_proxy_async_smem();
    mbar_expect_tx(&bars->k_full, p.pk * MC_PANEL);
    for (int i = 0; i < p.pk; ++i) tma_load_3d(sK + i * MC_PANEL, &tmK, &bars->k_full, i * 64, t0, h / (p.H / p.G));
    mbar_expect_tx(&bars->v_full, p.pv * MC_PANEL);
    for (int i = 0; i < p.pv; ++i) tma_load_3d(sV + i * MC_PANEL, &tmV, &bars->v_full, i * 64, t0, h);
  }
  if (warp == 1) {
    tmem_alloc(&bars->tmem_slot, 512);
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
  const uint64_t dk = make_smem_desc(smem_u32(sK), 16, 1024);
  if (tid == 0 && ok) {
    tc_fence_after();
    const uint32_t idesc = make_idesc_bf16(128, MC_C, 0, 0);
    for (int k = 0; k < (p.dim + 15) >> 4; ++k) {
      const int o = (k >> 2) * (MC_PANEL >> 4) + 2 * (k & 3);
      umma_bf16(tmem, dk + o, dk + o, idesc, k ? 1u : 0u);
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
    p.fk[idx * MC_C + t] = rk;
  }
  __syncthreads();
  ok = ok && mbar_wait(&bars->s_done, 0, abort_flag, p.err, ERR_WAIT_TMEM_FULL);
  ok = __all_sync(0xffffffffu, ok);
  // A below the diagonal, zeros above
  const float arow = sF[t], brow = beta * rk;
  if (ok) tc_fence_after();
#pragma unroll 1
  for (int b = 0; b < 2; ++b) {
    const int c0 = 64 * half + 32 * b;
    float* m = M + t * DC_PITCH + c0;
    if (!ok || c0 > (warp & 3) * 32 + 31) {
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
  join_blocks<16, 2, 2>(M, Y, tid);
  join_blocks<32, 2, 4>(M, Y, tid);
  join_blocks<64, 4, 4>(M, Y, tid);
  // rows of T diag(beta) and T diag(beta exp(F) fk) as heads and remainders
#pragma unroll 1
  for (int b = 0; b < 2; ++b) {
    const int c0 = 64 * half + 32 * b;
    uint32_t hi[2][16], lo[2][16];
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
      float m[4], s[4], f[4], r[4];
      ld4(M + t * DC_PITCH + c0 + i, m);
      ld4(sB + c0 + i, s);
      ld4(sF + c0 + i, f);
      ld4(sR + c0 + i, r);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[e] *= m[e];
        r[e] *= s[e] * ex2_approx(f[e]);
      }
      split_pack(s[0], s[1], hi[0][i >> 1], lo[0][i >> 1]);
      split_pack(s[2], s[3], hi[0][(i >> 1) + 1], lo[0][(i >> 1) + 1]);
      split_pack(r[0], r[1], hi[1][i >> 1], lo[1][i >> 1]);
      split_pack(r[2], r[3], hi[1][(i >> 1) + 1], lo[1][(i >> 1) + 1]);
    }
#pragma unroll
    for (int w = 0; w < 2; ++w) {
      tmem_st_32x16(ta + 128 * w + (c0 >> 1), hi[w]);
      tmem_st_32x16(ta + 128 * w + 64 + (c0 >> 1), lo[w]);
    }
  }
  tmem_st_wait();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (tid == 0) {
    const bool vok = mbar_wait(&bars->v_full, 0, abort_flag, p.err, ERR_WAIT_TMA_FULL);
    if (ok && vok) {
      tc_fence_after();
      const uint32_t idesc_v = make_idesc_bf16(128, p.vpad, 0, 1), idesc_k = make_idesc_bf16(128, (p.dim + 15) & ~15, 0, 1);
      const uint64_t dv = make_smem_desc(smem_u32(sV), MC_PANEL, 1024), dkm = make_smem_desc(smem_u32(sK), MC_PANEL, 1024);
      const int steps = (n + 15) >> 4;
      for (int part = 0; part < 2; ++part)
        for (int k = 0; k < steps; ++k) {
          umma_bf16_ts(tmem + 256, tmem + 64 * part + k * 8, dv + k * 128, idesc_v, (part || k) ? 1u : 0u);
          umma_bf16_ts(tmem + 384, tmem + 128 + 64 * part + k * 8, dkm + k * 128, idesc_k, (part || k) ? 1u : 0u);
        }
      umma_commit(&bars->uw_done);
    } else {
      bars->abort_flag = 1;
    }
  }
  ok = mbar_wait(&bars->uw_done, 0, abort_flag, p.err, ERR_WAIT_TMEM_FULL);
  if (__all_sync(0xffffffffu, ok)) {
    tc_fence_after();
    float* u = p.u0 + (idx * MC_C + t) * p.vpad;
    for (int v0 = 16 * half; v0 < p.vpad; v0 += 32) {
      uint32_t r[16];
      tmem_ld_32x16(ta + 256 + v0, r);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 16; i += 4) *reinterpret_cast<uint4*>(u + v0 + i) = make_uint4(r[i], r[i + 1], r[i + 2], r[i + 3]);
    }
    const size_t wrow = (idx * MC_C + t) * p.dim;
    for (int c0 = 16 * half; c0 < p.dim; c0 += 32) {
      uint32_t r[16], hi[8], lo[8];
      tmem_ld_32x16(ta + 384 + c0, r);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 8; ++i) split_pack(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1]), hi[i], lo[i]);
#pragma unroll
      for (int q = 0; q < 2; ++q)
        if (c0 + 8 * q < p.dim) {
          *reinterpret_cast<uint4*>(p.w_hi + wrow + c0 + 8 * q) = make_uint4(hi[4 * q], hi[4 * q + 1], hi[4 * q + 2], hi[4 * q + 3]);
          *reinterpret_cast<uint4*>(p.w_lo + wrow + c0 + 8 * q) = make_uint4(lo[4 * q], lo[4 * q + 1], lo[4 * q + 2], lo[4 * q + 3]);
        }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// ------------------------------------------------------------------------------------------------ recurrence over chunks
struct DeltaStateBars {
  uint64_t w_full, k_full;                     // W (head, remainder) and keys of a chunk have landed
  uint64_t s_ready, x_done, u_ready, d_done;   // state in shared memory; W S formed; weighted U in shared memory; K^T U formed
  uint64_t s_free;                             // the state's tile has been copied out
  uint32_t tmem_slot;
  int abort_flag;
};

// CTA: VB value columns of one head of one sequence.  Warps 0-3: thread = token row of W S and key row of the state; warp 4: MMAs; warp 5:
// copies.
template <int VB>
__global__ void __launch_bounds__(192, 1)
delta_state_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmWh, const __grid_constant__ CUtensorMap tmWl,
                   const __grid_constant__ CUtensorMap tmSh, const __grid_constant__ CUtensorMap tmSl, const DeltaChunkParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int SPANEL = VB * 128;
  DeltaStateBars* bars = reinterpret_cast<DeltaStateBars*>(smem);
  uint8_t* sWh = smem + 1024;
  uint8_t* sWl = sWh + p.pk * MC_PANEL;
  uint8_t* sK = sWl + p.pk * MC_PANEL;         // two panels: the product's 128 rows are key columns
  uint8_t* sUh = sK + 2 * MC_PANEL;            // token rows
  uint8_t* sUl = sUh + MC_PANEL;
  uint8_t* sSh = sUl + MC_PANEL;               // value rows, key columns
  uint8_t* sSl = sSh + p.pk * SPANEL;
  volatile int* abort_flag = &bars->abort_flag;
  const int v0 = blockIdx.x * VB, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int4 sq = p.seqs[blockIdx.z];
  const int c0 = sq.x, nc = sq.y, hk = h / (p.H / p.G);
  auto load_w = [&](int c) {
    const int plane = (c0 + c) * p.H + h;
    mbar_expect_tx(&bars->w_full, 2 * p.pk * MC_PANEL);
    for (int i = 0; i < p.pk; ++i) {
      tma_load_3d(sWh + i * MC_PANEL, &tmWh, &bars->w_full, i * 64, 0, plane);
      tma_load_3d(sWl + i * MC_PANEL, &tmWl, &bars->w_full, i * 64, 0, plane);
    }
  };
  auto load_k = [&](int c) {
    mbar_expect_tx(&bars->k_full, p.pk * MC_PANEL);
    for (int i = 0; i < p.pk; ++i) tma_load_3d(sK + i * MC_PANEL, &tmK, &bars->k_full, i * 64, p.chunks[c0 + c].x, hk);
  };
  if (tid == 160) {
    mbar_init(&bars->w_full, 1);
    mbar_init(&bars->k_full, 1);
    mbar_init(&bars->s_ready, 4);
    mbar_init(&bars->x_done, 1);
    mbar_init(&bars->u_ready, 4);
    mbar_init(&bars->d_done, 1);
    mbar_init(&bars->s_free, 1);
    bars->abort_flag = 0;
    fence_barrier_init();
    fence_proxy_async_smem();
    load_w(0);
    load_k(0);
  }
  if (warp == 4) {
    tmem_alloc(&bars->tmem_slot, 64);
    tmem_relinquish();
  }
  for (int i = tid; i < p.pk * SPANEL / 8; i += 192) reinterpret_cast<uint4*>(sSh)[i] = make_uint4(0u, 0u, 0u, 0u);   // both tiles; columns past dim stay zero
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_slot, tx = tmem, td = tmem + VB;
  auto wait = [&](uint64_t* bar, uint32_t ph, int code) { return mbar_wait(bar, ph, abort_flag, p.err, code); };
  if (warp == 4) {
    if (lane == 0) {
      const int ks = (p.dim + 15) >> 4;
      const uint32_t idesc_x = make_idesc_bf16(128, VB, 0, 0), idesc_d = make_idesc_bf16(128, VB, 1, 1);
      const uint64_t dwh = make_smem_desc(smem_u32(sWh), 16, 1024), dwl = make_smem_desc(smem_u32(sWl), 16, 1024), dsh = make_smem_desc(smem_u32(sSh), 16, 1024),
                     dsl = make_smem_desc(smem_u32(sSl), 16, 1024), dk = make_smem_desc(smem_u32(sK), MC_PANEL, 1024),
                     duh = make_smem_desc(smem_u32(sUh), MC_PANEL, 1024), dul = make_smem_desc(smem_u32(sUl), MC_PANEL, 1024);
      for (int c = 0; c < nc; ++c) {
        const uint32_t ph = c & 1;
        if (!wait(&bars->w_full, ph, ERR_WAIT_TMA_FULL) || !wait(&bars->s_ready, ph, ERR_WAIT_TMEM_FULL)) break;
        tc_fence_after();
        for (int part = 0; part < 3; ++part) {          // heads, then one remainder each
          const uint64_t dw = part == 2 ? dwl : dwh, ds = part == 1 ? dsl : dsh;
          for (int k = 0; k < ks; ++k)
            umma_bf16(tx, dw + (k >> 2) * (MC_PANEL >> 4) + 2 * (k & 3), ds + (k >> 2) * (SPANEL >> 4) + 2 * (k & 3), idesc_x, (part || k) ? 1u : 0u);
        }
        umma_commit(&bars->x_done);
        const int steps = (p.chunks[c0 + c].y + 15) >> 4;
        if (!wait(&bars->k_full, ph, ERR_WAIT_TMA_FULL) || !wait(&bars->u_ready, ph, ERR_WAIT_TMEM_FULL)) break;
        tc_fence_after();
        for (int part = 0; part < 2; ++part)
          for (int k = 0; k < steps; ++k) umma_bf16(td, dk + k * 128, (part ? dul : duh) + k * 128, idesc_d, (part || k) ? 1u : 0u);
        umma_commit(&bars->d_done);
      }
    }
  } else if (warp == 5) {
    if (lane == 0) {
      int w = 1, k = 1;                                  // loads issued
      bool ok = true;
      for (int c = 0; c < nc && ok; ++c) {
        const uint32_t ph = c & 1;
        ok = wait(&bars->s_ready, ph, ERR_WAIT_TMEM_FULL);
        if (!ok) break;
        const int row = ((c0 + c) * p.H + h) * p.vpad + v0;
        for (int i = 0; i < p.pk; ++i) {
          tma_store_2d(&tmSh, sSh + i * SPANEL, i * 64, row);
          tma_store_2d(&tmSl, sSl + i * SPANEL, i * 64, row);
        }
        bulk_commit_group();
        ok = wait(&bars->x_done, ph, ERR_WAIT_TMEM_FULL);
        if (ok && c + 1 < nc) {
          load_w(c + 1);
          ++w;
        }
        bulk_wait_read_all();
        mbar_arrive(&bars->s_free);
        ok = ok && wait(&bars->d_done, ph, ERR_WAIT_TMEM_FULL);
        if (ok && c + 1 < nc) {
          load_k(c + 1);
          ++k;
        }
      }
      bulk_wait_all();
      const unsigned long long begin = globaltimer_ns();   // a copy in flight has to land before the CTA ends
      while (!(mbar_try_wait(&bars->w_full, (w - 1) & 1) && mbar_try_wait(&bars->k_full, (k - 1) & 1)) && globaltimer_ns() - begin < WAIT_LIMIT_NS) {}
    }
  } else {
    const uint32_t lane_addr = static_cast<uint32_t>(warp * 32) << 16;
    const int r = tid;                                   // token of the chunk and key row of the state
    float* st = p.state + ((static_cast<size_t>(sq.z) * p.H + h) * p.dim + r) * p.ldv + v0;
    float S[VB];
#pragma unroll
    for (int v = 0; v < VB; ++v) S[v] = sq.w != 0 && r < p.dim && v0 + v < p.vdim ? st[v] : 0.f;
    auto put_state = [&]() {
      if (r < p.dim) {
        const int at = (r >> 6) * SPANEL + (r & 7) * 2, piece = (r & 63) >> 3;
#pragma unroll
        for (int v = 0; v < VB; ++v) {
          const __nv_bfloat16 hi = f2bf(S[v]);
          const int off = at + v * 128 + ((piece ^ (v & 7)) << 4);
          *reinterpret_cast<__nv_bfloat16*>(sSh + off) = hi;
          *reinterpret_cast<__nv_bfloat16*>(sSl + off) = f2bf(S[v] - bf2f(hi));
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->s_ready);
    };
    put_state();
    for (int c = 0; c < nc; ++c) {
      const uint32_t ph = c & 1;
      const int4 ck = p.chunks[c0 + c];
      const size_t idx = static_cast<size_t>(c0 + c) * p.H + h;
      float u[VB];
      const float* src = p.u0 + (idx * MC_C + r) * p.vpad + v0;
#pragma unroll
      for (int v = 0; v < VB; v += 4) {
        const float4 x = *reinterpret_cast<const float4*>(src + v);
        u[v] = x.x; u[v + 1] = x.y; u[v + 2] = x.z; u[v + 3] = x.w;
      }
      const float F = p.prefix[idx * MC_C + r], Fend = p.prefix[idx * MC_C + MC_C - 1], fk = p.fk[idx * MC_C + r];
      bool ok = wait(&bars->x_done, ph, ERR_WAIT_TMEM_FULL);
      if (!__all_sync(0xffffffffu, ok)) break;
      tc_fence_after();
#pragma unroll
      for (int b = 0; b < VB; b += 16) {
        uint32_t x[16];
        tmem_ld_32x16(tx + lane_addr + b, x);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) u[b + i] -= __uint_as_float(x[i]);
      }
      const float f = r < ck.y ? expf(Fend - F) * fk : 0.f;
#pragma unroll
      for (int q = 0; q < VB / 8; ++q) {                 // pieces of eight values of the token's row
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) split_pack(u[8 * q + 2 * i] * f, u[8 * q + 2 * i + 1] * f, hi[i], lo[i]);
        const int off = r * 128 + ((q ^ (r & 7)) << 4);
        *reinterpret_cast<uint4*>(sUh + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(sUl + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->u_ready);
      if (r < ck.y) {
        __nv_bfloat16* dst = p.u + static_cast<size_t>(ck.x + r) * p.ld_u + h * p.vdim + v0;
#pragma unroll
        for (int q = 0; q < VB / 8; ++q)
          if (v0 + 8 * q < p.vdim)
            *reinterpret_cast<uint4*>(dst + 8 * q) = make_uint4(pack_bf16x2(u[8 * q], u[8 * q + 1]), pack_bf16x2(u[8 * q + 2], u[8 * q + 3]),
                                                                pack_bf16x2(u[8 * q + 4], u[8 * q + 5]), pack_bf16x2(u[8 * q + 6], u[8 * q + 7]));
      }
      ok = wait(&bars->d_done, ph, ERR_WAIT_TMEM_FULL);
      if (!__all_sync(0xffffffffu, ok)) break;
      tc_fence_after();
      const float a = expf(Fend);
#pragma unroll
      for (int b = 0; b < VB; b += 16) {
        uint32_t x[16];
        tmem_ld_32x16(td + lane_addr + b, x);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) S[b + i] = a * S[b + i] + __uint_as_float(x[i]);
      }
      if (c + 1 < nc) {
        ok = wait(&bars->s_free, ph, ERR_WAIT_TMEM_FULL);
        if (!__all_sync(0xffffffffu, ok)) break;
        put_state();
      } else if (r < p.dim) {
#pragma unroll
        for (int v = 0; v < VB; ++v)
          if (v0 + v < p.vdim) st[v] = S[v];
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 4) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, 64);
  }
}

// bf16 [rows, cols]; box: `box_rows` rows x 64 columns, 128-byte swizzle (as a single plane)
static int make_tmap_rows2(CUtensorMap* out, const void* base, uint64_t cols, uint64_t rows, uint32_t box_rows) {
  typedef CUresult (*Fn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*, const cuuint32_t*,
                         CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
  static Fn enc = nullptr;
  if (!enc) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) return -1;
    enc = reinterpret_cast<Fn>(ptr);
  }
  if ((reinterpret_cast<uintptr_t>(base) & 15) || (cols & 7)) return -2;
  cuuint64_t dims[2] = {cols, rows}, strides[1] = {cols * 2};
  cuuint32_t box[2] = {64, box_rows}, estr[2] = {1, 1};
  return enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : -3;
}

static int dc_smem_chunk(int pk, int pv) { return 1024 + 1024 + (pk + pv) * MC_PANEL + (MC_C * DC_PITCH + 64 * DC_YPITCH + 5 * MC_C) * 4; }
static int dc_smem_state(int pk, int vb) { return 1024 + 1024 + (2 * pk + 2 + 2) * MC_PANEL + 2 * pk * vb * 128; }

template <int VB>
static int launch_delta_state(const CUtensorMap* tm, const DeltaChunkParams& p, int n_seqs, cudaStream_t st) {
  const int smem = dc_smem_state(p.pk, VB);
  if (cudaFuncSetAttribute(delta_state_kernel<VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
  delta_state_kernel<VB><<<dim3(p.vpad / VB, p.H, n_seqs), 192, smem, st>>>(tm[0], tm[1], tm[2], tm[3], tm[4], p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
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
  const int vb = p.vpad % 32 ? 16 : 32;
  const uint64_t planes = static_cast<uint64_t>(n_chunks) * p.H;
  if (planes * p.vpad > 0x7fffffffull) return -1;
  CUtensorMap tm[5], tv;
  int rc = make_tmap_planes(&tm[0], k, p.dim, T, p.G, ld, p.dim, MC_C);
  if (!rc) rc = make_tmap_planes(&tv, v, p.vdim, T, p.H, ld, p.vdim, MC_C);
  if (!rc) rc = make_tmap_planes(&tm[1], p.w_hi, p.dim, MC_C, planes, p.dim, static_cast<uint64_t>(MC_C) * p.dim, MC_C);
  if (!rc) rc = make_tmap_planes(&tm[2], p.w_lo, p.dim, MC_C, planes, p.dim, static_cast<uint64_t>(MC_C) * p.dim, MC_C);
  if (!rc) rc = make_tmap_rows2(&tm[3], p.s_hi, p.dim, planes * p.vpad, vb);
  if (!rc) rc = make_tmap_rows2(&tm[4], p.s_lo, p.dim, planes * p.vpad, vb);
  if (rc) return rc;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (parts & 1) {
    const int smem = dc_smem_chunk(p.pk, p.pv);
    if (cudaFuncSetAttribute(delta_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
    delta_chunk_kernel<<<dim3(p.H, n_chunks), 256, smem, st>>>(tm[0], tv, p);
    if (cudaGetLastError() != cudaSuccess) return -2;
  }
  if (parts & 2) return vb == 32 ? launch_delta_state<32>(tm, p, n_seqs, st) : launch_delta_state<16>(tm, p, n_seqs, st);
  return 0;
}
