// Matrix memories over packed prompts, in chunks of 128 tokens on the 5th-generation tensor cores.
//
// A memory S_t = a_t S_(t-1) + b_t k_t v_t^T with one scalar pair per head and token is a product inside a chunk and a short
// recurrence between chunks.  With F the running sum of log a inside a chunk and i = log b:
//   chunk_state : U = sum_j exp(F_end - F_j + i_j - m_loc) k_j v_j^T                              per (chunk, head), in parallel
//   chunk_scan  : S before every chunk, S <- exp(F_end + m - m') S + exp(m_loc - m') U             per (sequence, head)
//   chunk_out   : o_t = sum_(j <= t) exp(F_t - F_j + i_j - m_t) (q_t . k_j) v_j + exp(F_t + m - m_t) S^T q_t
// The delta rule's u_j (delta_chunk.cu) take the place of v_j in chunk_out, with i = 0 and F from that file's kernels; keys and queries are
// made unit vectors by factors on the weights, and the read-outs are normed and gated per head.
// A fixed decay has i = 0 and needs no maxima m.  A gated memory carries the running maximum m (starting at 0) and its
// normaliser n, which rides along as one more value column of ones.
// Decays, gates, maxima, sums and the carried state are fp32.  Operands that stem from the state or carry a decay (S and the
// weighted keys) enter the products as a bf16 head plus a bf16 remainder.
// Between the kernels a state is stored transposed, [value rows][key columns], as chunk_out reads it.
#include "memory_chunk.cuh"

namespace b200 {

struct ChunkParams {
  int H, dim, vdim;
  int dimp, vpad, vrows;          // key columns padded to eight; value rows padded to 16, plus 16 for the normaliser
  int pk, pv;                     // 64-column panels
  int ldv, ld_in, ld_out, gate_t, gate_h;   // gate_t, gate_h: strides of `gates` per token and per gate
  float qscale, cap, eps;
  const int4* chunks;             // {first token, tokens, sequence, cache row if it is the first of a continued sequence, -1 of a fresh one, -2}
  const int4* seqs;               // {first chunk, chunks, cache row, first position}
  const float* log2_decay;        // fixed decay: [H]
  const float* gates;             // gated: raw projections [T, 2H] (strided), log input | log forget
  const float* gate_bias;         // [2H]
  float* u;                       // [chunks * H, vrows, dimp]
  float2* stat;                   // [chunks * H] {m_loc, F_end}
  __nv_bfloat16 *s_hi, *s_lo;     // [chunks * H, vpad, dimp]
  float* n_before;                // gated: [chunks * H, dimp] normaliser before each chunk
  float* m_before;                // [chunks * H]
  float* m_init;                  // [sequences * H]
  // DELTA
  int group, ld_g;                // value heads per key head; pitch of the output gate's rows
  const float *prefix, *fk;       // [chunks * H, 128] running sum of log decays; factor that makes the key a unit vector
  float* state;                   // cache [rows, H, dim, ldv]
  float* stab;                    // cache [rows, H, dim + 1]
  const __nv_bfloat16* gate_out;  // gated: output gate, head h at column h * vdim, pitch ld_g
  const float* norm_w;
  __nv_bfloat16* out;             // [T, ld_out]
  int* err;
};

struct ChunkBars {
  uint64_t qk_full, v_full, o_done;
  uint32_t tmem_slot;
  int abort_flag;
  float red[16];
};

// log input and log forget gate of a token
__device__ __forceinline__ void token_gates(const ChunkParams& p, int t, int h, float& li, float& lf) {
  const float zi = p.gates[static_cast<size_t>(t) * p.gate_t + static_cast<size_t>(h) * p.gate_h] + p.gate_bias[h];
  const float zf = p.gates[static_cast<size_t>(t) * p.gate_t + static_cast<size_t>(p.H + h) * p.gate_h] + p.gate_bias[p.H + h];
  li = p.cap * tanhf(zi / p.cap);
  const float z = p.cap * tanhf(zf / p.cap);
  lf = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

// ------------------------------------------------------------------------------------------------ states of single chunks
template <bool GATED>
__global__ void __launch_bounds__(256)
chunk_state_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const ChunkParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  ChunkBars* bars = reinterpret_cast<ChunkBars*>(smem);
  uint8_t* sKh = smem + 1024;                  // two panels: the product's 128 rows are key columns
  uint8_t* sKl = sKh + 2 * MC_PANEL;
  uint8_t* sV = sKl + 2 * MC_PANEL;
  uint8_t* sOne = sV + p.pv * MC_PANEL;        // gated: a column of ones
  volatile int* abort_flag = &bars->abort_flag;
  // thread: token j of the chunk (later: key column j), half of the row's columns
  const int h = blockIdx.x, ch = blockIdx.y, j = threadIdx.x & 127, half = threadIdx.x >> 7, warp = threadIdx.x >> 5;
  const int4 c = p.chunks[ch];
  const int t0 = c.x, n = c.y;
  if (threadIdx.x == 0) {
    mbar_init(&bars->qk_full, 1);
    mbar_init(&bars->v_full, 1);
    mbar_init(&bars->o_done, 1);
    bars->abort_flag = 0;
    fence_barrier_init();
    fence_proxy_async_smem();
    mbar_expect_tx(&bars->qk_full, p.pk * MC_PANEL);
    for (int i = 0; i < p.pk; ++i) tma_load_3d(sKh + i * MC_PANEL, &tmK, &bars->qk_full, i * 64, t0, h);
    mbar_expect_tx(&bars->v_full, p.pv * MC_PANEL);
    for (int i = 0; i < p.pv; ++i) tma_load_3d(sV + i * MC_PANEL, &tmV, &bars->v_full, i * 64, t0, h);
  }
  uint32_t cols = 32;
  while (cols < static_cast<uint32_t>(p.vrows)) cols <<= 1;
  if (warp == 1) {
    tmem_alloc(&bars->tmem_slot, cols);
    tmem_relinquish();
  }
  // weights
  float w;
  const size_t idx = static_cast<size_t>(ch) * p.H + h;
  if constexpr (GATED) {
    float li = -INFINITY, lf = 0.f;
    if (j < n) token_gates(p, t0 + j, h, li, lf);
    const float F = chunk_prefix<false>(lf, bars->red);
    if (j == MC_C - 1) bars->red[8] = F;       // tokens past the end add nothing
    __syncthreads();
    const float Fend = bars->red[8], e = Fend - F + li;
    const float m = chunk_prefix<true>(e, bars->red);
    if (j == MC_C - 1) bars->red[9] = m;
    __syncthreads();
    const float mloc = bars->red[9];
    w = j < n ? expf(e - mloc) : 0.f;
    if (threadIdx.x == 0) {
      p.stat[idx] = make_float2(mloc, Fend);
      if (c.w > -2) p.m_init[static_cast<size_t>(c.z) * p.H + h] = c.w < 0 ? 0.f : p.stab[(static_cast<size_t>(c.w) * p.H + h) * (p.dim + 1) + p.dim];
    }
    for (int i = 4 * half; i < 4 * half + 4; ++i) {   // the row's pieces, ones in the first column
      const uint32_t one = i == 0 ? 0x3F80u : 0u;
      *reinterpret_cast<uint4*>(sOne + j * 128 + ((i ^ (j & 7)) << 4)) = make_uint4(one, 0u, 0u, 0u);
    }
  } else {
    w = j < n ? exp2f(p.log2_decay[h] * static_cast<float>(n - 1 - j)) : 0.f;
    if (threadIdx.x == 0) p.stat[idx] = make_float2(0.f, p.log2_decay[h] * static_cast<float>(n));
  }
  __syncthreads();
  const bool ok = mbar_wait(&bars->qk_full, 0, abort_flag, p.err, ERR_WAIT_TMA_FULL);
#pragma unroll 4
  for (int i = 8 * half; i < 8 * half + 8; ++i) {
    const int off = (i >> 3) * MC_PANEL + j * 128 + (((i & 7) ^ (j & 7)) << 4);
    uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
    if (w != 0.f && i < 8 * p.pk) {
      const uint4 k = *reinterpret_cast<const uint4*>(sKh + off);
      const float2 a = unpack_bf16x2(k.x), b = unpack_bf16x2(k.y), d = unpack_bf16x2(k.z), e = unpack_bf16x2(k.w);
      split_pack(a.x * w, a.y * w, hi.x, lo.x);
      split_pack(b.x * w, b.y * w, hi.y, lo.y);
      split_pack(d.x * w, d.y * w, hi.z, lo.z);
      split_pack(e.x * w, e.y * w, hi.w, lo.w);
    }
    *reinterpret_cast<uint4*>(sKh + off) = hi;
    *reinterpret_cast<uint4*>(sKl + off) = lo;
  }
  fence_proxy_async_smem();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_slot;
  if (threadIdx.x == 0) {
    const bool vok = mbar_wait(&bars->v_full, 0, abort_flag, p.err, ERR_WAIT_TMA_FULL);
    if (ok && vok) {
      tc_fence_after();
      const uint32_t idesc = make_idesc_bf16(128, p.vpad, 1, 1), idesc1 = make_idesc_bf16(128, 16, 1, 1);
      const uint64_t dv = make_smem_desc(smem_u32(sV), MC_PANEL, 1024), d1 = make_smem_desc(smem_u32(sOne), MC_PANEL, 1024);
      const int steps = (n + 15) >> 4;
      for (int part = 0; part < 2; ++part) {
        const uint64_t dk = make_smem_desc(smem_u32(part ? sKl : sKh), MC_PANEL, 1024);
        for (int t = 0; t < steps; ++t) {
          umma_bf16(tmem, dk + t * 128, dv + t * 128, idesc, (part || t) ? 1u : 0u);
          if constexpr (GATED) umma_bf16(tmem + p.vpad, dk + t * 128, d1 + t * 128, idesc1, (part || t) ? 1u : 0u);
        }
      }
      umma_commit(&bars->o_done);
    } else {
      bars->abort_flag = 1;
    }
  }
  if (mbar_wait(&bars->o_done, 0, abort_flag, p.err, ERR_WAIT_TMEM_FULL)) {
    tc_fence_after();
    float* u = p.u + idx * p.vrows * p.dimp + j;
    const uint32_t ta = tmem + (static_cast<uint32_t>((warp & 3) * 32) << 16);
    for (int v0 = 16 * half; v0 < p.vrows; v0 += 32) {
      uint32_t r[16];
      tmem_ld_32x16(ta + v0, r);
      tmem_ld_wait();
      if (j < p.dimp) {
#pragma unroll
        for (int i = 0; i < 16; ++i) u[static_cast<size_t>(v0 + i) * p.dimp] = __uint_as_float(r[i]);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, cols);
  }
}

// ------------------------------------------------------------------------------------------------ recurrence over chunks
// A thread carries four key columns of one value row through the chunks of a sequence.
template <bool GATED>
__global__ void __launch_bounds__(128)
chunk_scan_kernel(const ChunkParams p) {
  const int h = blockIdx.y;
  const int4 sq = p.seqs[blockIdx.z];
  const int c0 = sq.x, nc = sq.y, row = sq.z;
  const bool fresh = sq.w == 0;
  const int per = p.dimp >> 2, e = blockIdx.x * 128 + threadIdx.x;
  if (e >= per * p.vrows) return;
  const int v = e / per, d = 4 * (e - v * per);
  float* st = p.state + (static_cast<size_t>(row) * p.H + h) * p.dim * p.ldv;
  float* sb = GATED ? p.stab + (static_cast<size_t>(row) * p.H + h) * (p.dim + 1) : nullptr;
  const bool is_value = v < p.vdim, is_norm = GATED && v == p.vpad;
  float s[4] = {0.f, 0.f, 0.f, 0.f};
  if (!fresh) {
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (d + i < p.dim) {
        if (is_value) s[i] = st[static_cast<size_t>(d + i) * p.ldv + v];
        else if (is_norm) s[i] = sb[d + i];
      }
  }
  float m = GATED ? p.m_init[static_cast<size_t>(blockIdx.z) * p.H + h] : 0.f;
  const size_t pitch = static_cast<size_t>(p.vrows) * p.dimp, spitch = static_cast<size_t>(p.vpad) * p.dimp, at = static_cast<size_t>(v) * p.dimp + d;
  constexpr int U = 8;                         // chunks in flight
  for (int b = 0; b < nc; b += U) {
    float4 u[U];
    float2 f[U];
#pragma unroll
    for (int k = 0; k < U; ++k)
      if (b + k < nc) {
        const size_t idx = static_cast<size_t>(c0 + b + k) * p.H + h;
        u[k] = *reinterpret_cast<const float4*>(p.u + idx * pitch + at);
        f[k] = p.stat[idx];
      }
#pragma unroll
    for (int k = 0; k < U; ++k)
      if (b + k < nc) {
        const size_t idx = static_cast<size_t>(c0 + b + k) * p.H + h;
        if (!GATED || v < p.vpad) {
          uint2 hi, lo;
          split_pack(s[0], s[1], hi.x, lo.x);
          split_pack(s[2], s[3], hi.y, lo.y);
          *reinterpret_cast<uint2*>(p.s_hi + idx * spitch + at) = hi;
          *reinterpret_cast<uint2*>(p.s_lo + idx * spitch + at) = lo;
        } else if (is_norm) {
          *reinterpret_cast<float4*>(p.n_before + idx * p.dimp + d) = make_float4(s[0], s[1], s[2], s[3]);
        }
        float a, w = 1.f;
        if constexpr (GATED) {
          if (e == 0) p.m_before[idx] = m;
          const float mn = fmaxf(f[k].y + m, f[k].x);
          a = expf(f[k].y + m - mn);
          w = expf(f[k].x - mn);
          m = mn;
        } else {
          a = exp2f(f[k].y);
        }
        s[0] = a * s[0] + w * u[k].x;
        s[1] = a * s[1] + w * u[k].y;
        s[2] = a * s[2] + w * u[k].z;
        s[3] = a * s[3] + w * u[k].w;
      }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
    if (d + i < p.dim) {
      if (is_value) st[static_cast<size_t>(d + i) * p.ldv + v] = s[i];
      else if (is_norm) sb[d + i] = s[i];
    }
  if (GATED && e == 0) sb[p.dim] = m;
}

// ------------------------------------------------------------------------------------------------ outputs
enum MemoryKind { DECAY = 0, GATED = 1, DELTA = 2 };

struct ChunkOutBars {
  uint64_t qk_full, v_full, s_full, s_done, o_part, o_done, p_ready, final;
  uint32_t tmem_slot;
  int abort_flag;
  float red[8];
};

// Warps 0-7: token j = thread & 127 of the chunk, its columns shared by the two halves; warp 8: copies and MMAs.
// Shared memory is used twice so that two CTAs fit an SM: the values follow the keys once the scores are formed, the state's
// remainder follows its head once that product is done.  Tensor memory: scores, then bf16 weights over them; outputs at MC_C.
// KS: 16-column steps of the keys, known at compile time for common sizes (the issuing thread's address arithmetic would pace the
// products otherwise); 0: read from the parameters.
template <int KIND, int KS>
__global__ void __launch_bounds__(288, 2)
chunk_out_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                 const __grid_constant__ CUtensorMap tmSh, const __grid_constant__ CUtensorMap tmSl, const ChunkParams p, int tmem_cols) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  ChunkOutBars* bars = reinterpret_cast<ChunkOutBars*>(smem);
  float* gj = reinterpret_cast<float*>(smem + 512);      // [128] exponent of key j
  float* nsum = reinterpret_cast<float*>(smem + 1024);   // [2][128] partial n . q
  float* nb = reinterpret_cast<float*>(smem + 2048);     // [128] normaliser before the chunk
  const int spanel = p.vpad * 128;
  uint8_t* sQ = smem + 3072;
  uint8_t* sKV = sQ + p.pk * MC_PANEL;
  uint8_t* sS = sKV + max(p.pk, p.pv) * MC_PANEL;
  volatile int* abort_flag = &bars->abort_flag;
  const int h = blockIdx.x, ch = blockIdx.y, j = threadIdx.x & 127, half = threadIdx.x >> 7, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int4 c = p.chunks[ch];
  const int t0 = c.x, n = c.y;
  const size_t idx = static_cast<size_t>(ch) * p.H + h;
  const int hk = KIND == DELTA ? h / p.group : h;
  if (threadIdx.x == 256) {
    mbar_init(&bars->qk_full, 1);
    mbar_init(&bars->v_full, 1);
    mbar_init(&bars->s_full, 1);
    mbar_init(&bars->s_done, 1);
    mbar_init(&bars->o_part, 1);
    mbar_init(&bars->o_done, 1);
    mbar_init(&bars->p_ready, 8);
    mbar_init(&bars->final, 1);
    bars->abort_flag = 0;
    fence_barrier_init();
    fence_proxy_async_smem();
    mbar_expect_tx(&bars->qk_full, p.pk * 2 * MC_PANEL);
    for (int i = 0; i < p.pk; ++i) {
      tma_load_3d(sQ + i * MC_PANEL, &tmQ, &bars->qk_full, i * 64, t0, hk);
      tma_load_3d(sKV + i * MC_PANEL, &tmK, &bars->qk_full, i * 64, t0, hk);
    }
    mbar_expect_tx(&bars->s_full, p.pk * spanel);
    for (int i = 0; i < p.pk; ++i) tma_load_3d(sS + i * spanel, &tmSh, &bars->s_full, i * 64, 0, static_cast<int>(idx));
  }
  if (warp == 8) {
    __syncwarp();
    tmem_alloc(&bars->tmem_slot, tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_slot;
  if (warp == 8) {
    if (lane == 0) {
      const int ks = (p.dim + 15) >> 4;
      const uint64_t dq = make_smem_desc(smem_u32(sQ), 16, 1024), dk = make_smem_desc(smem_u32(sKV), 16, 1024), ds = make_smem_desc(smem_u32(sS), 16, 1024),
                     dv = make_smem_desc(smem_u32(sKV), MC_PANEL, 1024);
      const uint32_t idesc_s = make_idesc_bf16(128, MC_C, 0, 0), idesc_o = make_idesc_bf16(128, p.vpad, 0, 0), idesc_v = make_idesc_bf16(128, p.vpad, 0, 1);
      auto wait = [&](uint64_t* bar, uint32_t ph, int code) { return mbar_wait(bar, ph, abort_flag, p.err, code); };
      auto state_product = [&](uint32_t acc) {
        tc_fence_after();
        if constexpr (KS > 0) {
#pragma unroll
          for (int t = 0; t < KS; ++t)
            umma_bf16(tmem + MC_C, dq + ((t >> 2) * (MC_PANEL >> 4) + 2 * (t & 3)), ds + (t >> 2) * (spanel >> 4) + 2 * (t & 3), idesc_o, t ? 1u : acc);
          return;
        }
        for (int t = 0; t < ks; ++t)
          umma_bf16(tmem + MC_C, dq + (t >> 2) * (MC_PANEL >> 4) + 2 * (t & 3), ds + (t >> 2) * (spanel >> 4) + 2 * (t & 3), idesc_o, (acc || t) ? 1u : 0u);
      };
      bool ok = wait(&bars->qk_full, 0, ERR_WAIT_TMA_FULL);
      if (ok) {
        tc_fence_after();
        if constexpr (KS > 0) {
#pragma unroll
          for (int t = 0; t < KS; ++t) umma_bf16(tmem, dq + ((t >> 2) * (MC_PANEL >> 4) + 2 * (t & 3)), dk + ((t >> 2) * (MC_PANEL >> 4) + 2 * (t & 3)), idesc_s, t ? 1u : 0u);
        } else {
          for (int t = 0; t < ks; ++t) {
            const int o = (t >> 2) * (MC_PANEL >> 4) + 2 * (t & 3);
            umma_bf16(tmem, dq + o, dk + o, idesc_s, t ? 1u : 0u);
          }
        }
        umma_commit(&bars->s_done);
        ok = wait(&bars->s_full, 0, ERR_WAIT_TMA_FULL);
      }
      if (ok) {
        state_product(0u);
        umma_commit(&bars->o_part);
        ok = wait(&bars->s_done, 0, ERR_WAIT_TMEM_FULL);          // the keys have been read
      }
      if (ok) {
        mbar_expect_tx(&bars->v_full, p.pv * MC_PANEL);
        for (int i = 0; i < p.pv; ++i) tma_load_3d(sKV + i * MC_PANEL, &tmV, &bars->v_full, i * 64, t0, h);
        ok = wait(&bars->o_part, 0, ERR_WAIT_TMEM_FULL);          // the state's head has been read
        if (ok) {
          mbar_expect_tx(&bars->s_full, p.pk * spanel);
          for (int i = 0; i < p.pk; ++i) tma_load_3d(sS + i * spanel, &tmSl, &bars->s_full, i * 64, 0, static_cast<int>(idx));
          ok = wait(&bars->s_full, 1, ERR_WAIT_TMA_FULL);
        }
        if (ok) {
          state_product(1u);
          umma_commit(&bars->o_done);
        }
        const bool vok = wait(&bars->v_full, 0, ERR_WAIT_TMA_FULL);   // in any case: the copy has to land before the CTA ends
        ok = ok && vok && wait(&bars->p_ready, 0, ERR_WAIT_TMEM_FULL);
      }
      if (ok) {
        tc_fence_after();
#pragma unroll
        for (int t = 0; t < MC_C / 16; ++t) umma_bf16_ts(tmem + MC_C, tmem + t * 8, dv + t * 128, idesc_v, 1u);
        umma_commit(&bars->final);
      } else {
        bars->abort_flag = 1;
        // a copy in flight has to land before the CTA ends
        const unsigned long long begin = globaltimer_ns();
        while (!(mbar_try_wait(&bars->qk_full, 0) && mbar_try_wait(&bars->s_full, 0)) && globaltimer_ns() - begin < WAIT_LIMIT_NS) {}
      }
    }
  } else {
    // exponents of this thread's row (and, as a key, of its column)
    float arow, einter, mrow = 0.f;
    if constexpr (KIND == GATED) {
      float li = -INFINITY, lf = 0.f;
      if (j < n) token_gates(p, t0 + j, h, li, lf);
      if (threadIdx.x < p.dim) nb[threadIdx.x] = p.n_before[idx * p.dimp + threadIdx.x];
      const float F = chunk_prefix<false>(lf, bars->red);
      const float pm = chunk_prefix<true>(li - F, bars->red);
      const float mb = p.m_before[idx];
      mrow = F + fmaxf(mb, pm);
      arow = (F - mrow) * LOG2E;
      einter = expf(F + mb - mrow);
      gj[j] = (li - F) * LOG2E;
    } else if constexpr (KIND == DELTA) {
      const float F = p.prefix[idx * MC_C + j];
      arow = F * LOG2E;
      gj[j] = -arow;
      nb[j] = p.fk[idx * MC_C + j];
      einter = exp2f(arow);
    } else {
      const float ld = p.log2_decay[h];
      arow = ld * static_cast<float>(j);
      gj[j] = -arow;
      einter = exp2f(ld * static_cast<float>(j + 1));
    }
    einter *= p.qscale;
    float qscale = p.qscale;
    named_barrier_sync(1, 256);
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t ts = tmem + lane_addr, to = ts + MC_C;
    float nq = 0.f;
    uint32_t packed[2][16];
    bool ok = mbar_wait(&bars->s_done, 0, abort_flag, p.err, ERR_WAIT_TMEM_FULL);
    if (ok) tc_fence_after();
    if constexpr (KIND == DELTA) {                    // unit vectors: factor of this row's query, half of its columns each
      float qq = 0.f;
      if (ok && mbar_wait(&bars->qk_full, 0, abort_flag, p.err, ERR_WAIT_TMA_FULL) && half < p.pk) {
#pragma unroll 4
        for (int i = 0; i < 8; ++i) {
          float q[8];
          ld8(reinterpret_cast<const __nv_bfloat16*>(sQ + half * MC_PANEL + j * 128 + ((i ^ (j & 7)) << 4)), q);
#pragma unroll
          for (int e = 0; e < 8; ++e) qq += q[e] * q[e];
        }
      }
      nsum[half * MC_C + j] = qq;
      named_barrier_sync(1, 256);
      const float fq = 1.f / sqrtf(nsum[j] + nsum[MC_C + j] + 1e-6f);
      qscale *= fq;
      einter *= fq;
    }
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int c0 = 32 * half + 64 * b;
      if (!ok || c0 > (warp & 3) * 32) {              // keys after every token of this warp
#pragma unroll
        for (int i = 0; i < 16; ++i) packed[b][i] = 0u;
      } else {
        uint32_t v[32];
        tmem_ld_32x32(ts + c0, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          const float4 g = *reinterpret_cast<const float4*>(gj + c0 + i);
          float w[4] = {g.x, g.y, g.z, g.w}, fk[4] = {1.f, 1.f, 1.f, 1.f};
          if constexpr (KIND == DELTA) ld4(nb + c0 + i, fk);
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            w[k] = c0 + i + k <= j ? __uint_as_float(v[i + k]) * qscale * ex2_approx(arow + w[k]) * fk[k] : 0.f;
            nq += w[k];
          }
          packed[b][i >> 1] = pack_bf16x2(w[0], w[1]);
          packed[b][(i >> 1) + 1] = pack_bf16x2(w[2], w[3]);
        }
      }
    }
    if constexpr (KIND == GATED) {
      // the state's part of n . q: this half's 64 key columns
      if (ok && mbar_wait(&bars->qk_full, 0, abort_flag, p.err, ERR_WAIT_TMA_FULL) && half < p.pk) {
        float d = 0.f;
        const int cols = min(64, p.dim - 64 * half);
#pragma unroll 4
        for (int i = 0; i < 8; ++i) {
          if (8 * i >= cols) break;
          float q[8];
          ld8(reinterpret_cast<const __nv_bfloat16*>(sQ + half * MC_PANEL + j * 128 + ((i ^ (j & 7)) << 4)), q);
          const float4 a = *reinterpret_cast<const float4*>(nb + 64 * half + 8 * i), e = *reinterpret_cast<const float4*>(nb + 64 * half + 8 * i + 4);
          d += q[0] * a.x + q[1] * a.y + q[2] * a.z + q[3] * a.w + q[4] * e.x + q[5] * e.y + q[6] * e.z + q[7] * e.w;
        }
        nq += d * einter;
      }
      nsum[half * MC_C + j] = nq;
    }
    tc_fence_before();
    named_barrier_sync(1, 256);                       // all scores have been read: the weights may lie over them
    tc_fence_after();
    if (ok) {
#pragma unroll
      for (int b = 0; b < 2; ++b) tmem_st_32x16(ts + 16 * half + 32 * b, packed[b]);
      ok = mbar_wait(&bars->o_done, 0, abort_flag, p.err, ERR_WAIT_TMEM_FULL);
    }
    if (ok) {
      tc_fence_after();
#pragma unroll 1
      for (int c0 = 32 * half; c0 < p.vpad; c0 += 64) {       // up to 16 unused columns behind the last
        uint32_t v[32];
        tmem_ld_32x32(to + c0, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * einter);
        tmem_st_32x32(to + c0, v);
      }
      tmem_st_wait();
    }
    tc_fence_before();
    __syncwarp();
    if (lane == 0) mbar_arrive(&bars->p_ready);
    if (ok && mbar_wait(&bars->final, 0, abort_flag, p.err, ERR_WAIT_TMEM_FULL)) {
      tc_fence_after();
      const bool live = j < n;
      const size_t t = static_cast<size_t>(t0) + (live ? j : 0);
      __nv_bfloat16* orow = p.out + t * p.ld_out + h * p.vdim;
      float f = 1.f;
      if constexpr (KIND == GATED) f = 1.f / (fmaxf(fabsf(nsum[j] + nsum[MC_C + j]), expf(-mrow)) + 1e-6f);
      if constexpr (KIND != DECAY) {
        float ss = 0.f;
#pragma unroll 1
        for (int c0 = 0; c0 < p.vpad; c0 += 16) {     // padding columns are zero
          uint32_t v[16];
          tmem_ld_32x16(to + c0, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const float o = __uint_as_float(v[i]) * f;
            ss += o * o;
          }
        }
        f /= sqrtf(ss / static_cast<float>(p.vdim) + p.eps);
      }
      const __nv_bfloat16* grow = KIND != DECAY ? p.gate_out + t * p.ld_g + h * p.vdim : nullptr;
      const float* nw = KIND == GATED ? p.norm_w + h * p.vdim : p.norm_w;
#pragma unroll 1
      for (int c0 = 16 * half; c0 < p.vpad; c0 += 32) {
        float g[2][8];
        if constexpr (KIND != DECAY) {                // requested before the accumulator is read
#pragma unroll
          for (int q = 0; q < 2; ++q)
            if (c0 + 8 * q < p.vdim) ld8(grow + c0 + 8 * q, g[q]);
        }
        uint32_t v[16];
        tmem_ld_32x16(to + c0, v);
        tmem_ld_wait();
        if (!live) continue;
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          if (c0 + 8 * q >= p.vdim) continue;
          float o[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) o[i] = __uint_as_float(v[8 * q + i]) * f;
          if constexpr (KIND != DECAY) {
            float w[8];
            ld8(nw + c0 + 8 * q, w);
#pragma unroll
            for (int i = 0; i < 8; ++i) o[i] *= w[i] * __fdividef(KIND == DELTA ? g[q][i] : 1.f, 1.f + __expf(-g[q][i]));
          }
          st8(orow + c0 + 8 * q, o);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 8) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, tmem_cols);
  }
}

template <int KIND, int KS>
static int launch_chunk_out(const CUtensorMap* tm, const ChunkParams& p, int n_chunks, int smem, int cols, cudaStream_t st) {
  if (cudaFuncSetAttribute(chunk_out_kernel<KIND, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
  chunk_out_kernel<KIND, KS><<<dim3(p.H, n_chunks), 288, smem, st>>>(tm[0], tm[1], tm[2], tm[3], tm[4], p, cols);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
template <int KIND>
static int dispatch_chunk_out(const CUtensorMap* tm, const ChunkParams& p, int n_chunks, int smem, int cols, cudaStream_t st) {
  switch ((p.dim + 15) / 16) {
    case 8: return launch_chunk_out<KIND, 8>(tm, p, n_chunks, smem, cols, st);
    case 6: return launch_chunk_out<KIND, 6>(tm, p, n_chunks, smem, cols, st);
    case 4: return launch_chunk_out<KIND, 4>(tm, p, n_chunks, smem, cols, st);
    default: return launch_chunk_out<KIND, 0>(tm, p, n_chunks, smem, cols, st);
  }
}

static int mc_smem_state(int pv, bool gated) { return 1024 + 1024 + (4 + pv + (gated ? 1 : 0)) * MC_PANEL; }
static int mc_smem_out(int pk, int pv, int vpad) { return 3072 + 1024 + (pk + (pk > pv ? pk : pv)) * MC_PANEL + pk * vpad * 128; }

}  // namespace b200

using namespace b200;

static int mc_vrows(int vdim, bool gated) { return ((vdim + 15) & ~15) + (gated ? 16 : 0); }

B200_API int b200_memory_chunk_supported(int dim, int vdim, int gated) {
  if (dim <= 0 || vdim <= 0 || (dim & 7) || (vdim & 7) || dim > 128 || mc_vrows(vdim, gated) > 256) return 0;
  const int pk = (dim + 63) / 64, pv = (vdim + 63) / 64, limit = 227 * 1024;
  return mc_smem_state(pv, gated) <= limit && mc_smem_out(pk, pv, (vdim + 15) & ~15) <= limit;
}

// q, k, v: columns of the packed step's projection rows [T, ld_in] (head h at column h dim / h vdim).  parts: 1 chunk states,
// 2 recurrence, 4 outputs (all of them in this order for a step).
B200_API int b200_memory_chunks(const void* q, const void* k, const void* v, const ChunkParams* Pp, int T, int n_chunks, int n_seqs, int parts,
                                void* stream, int* err) {
  ChunkParams p = *Pp;
  const bool gated = p.gates != nullptr;
  if (!b200_memory_chunk_supported(p.dim, p.vdim, gated) || T <= 0 || n_chunks <= 0 || n_chunks > 65535 || n_seqs <= 0 || n_seqs > 65535 ||
      p.H <= 0 || p.H > 65535 || (p.ld_in & 7) || (p.ld_out & 7) || (reinterpret_cast<uintptr_t>(p.out) & 15)) return -1;
  if (gated ? (!p.stab || !p.n_before || !p.norm_w || !p.gate_bias || ((reinterpret_cast<uintptr_t>(p.gate_out) | reinterpret_cast<uintptr_t>(p.norm_w)) & 15)) : !p.log2_decay) return -1;
  p.dimp = (p.dim + 7) & ~7;
  p.vpad = (p.vdim + 15) & ~15;
  p.vrows = mc_vrows(p.vdim, gated);
  p.pk = (p.dim + 63) / 64;
  p.pv = (p.vdim + 63) / 64;
  p.err = err;
  p.ld_g = p.ld_in;
  CUtensorMap tq, tk, tv, th, tl;
  int rc = make_tmap_planes(&tq, q, p.dim, T, p.H, p.ld_in, p.dim, MC_C);
  if (!rc) rc = make_tmap_planes(&tk, k, p.dim, T, p.H, p.ld_in, p.dim, MC_C);
  if (!rc) rc = make_tmap_planes(&tv, v, p.vdim, T, p.H, p.ld_in, p.vdim, MC_C);
  const uint64_t planes = static_cast<uint64_t>(n_chunks) * p.H;
  if (!rc) rc = make_tmap_planes(&th, p.s_hi, p.dim, p.vpad, planes, p.dimp, static_cast<uint64_t>(p.vpad) * p.dimp, p.vpad);
  if (!rc) rc = make_tmap_planes(&tl, p.s_lo, p.dim, p.vpad, planes, p.dimp, static_cast<uint64_t>(p.vpad) * p.dimp, p.vpad);
  if (rc) return rc;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const int sm1 = mc_smem_state(p.pv, gated), sm3 = mc_smem_out(p.pk, p.pv, p.vpad);
  int cols = 256;
  while (cols < MC_C + ((p.vpad + 31) & ~31)) cols <<= 1;
#define GO(G)                                                                                                          \
  {                                                                                                                    \
    if (cudaFuncSetAttribute(chunk_state_kernel<G>, cudaFuncAttributeMaxDynamicSharedMemorySize, sm1) != cudaSuccess) return -3; \
    if (parts & 1) chunk_state_kernel<G><<<dim3(p.H, n_chunks), 256, sm1, st>>>(tk, tv, p);                              \
    if (parts & 2) chunk_scan_kernel<G><<<dim3((p.vrows * (p.dimp / 4) + 127) / 128, p.H, n_seqs), 128, 0, st>>>(p);      \
    if (parts & 4) {                                                                                                    \
      const CUtensorMap tm[5] = {tq, tk, tv, th, tl};                                                                  \
      return dispatch_chunk_out<G ? GATED : DECAY>(tm, p, n_chunks, sm3, cols, st);                                     \
    }                                                                                                                  \
  }
  if (gated) GO(true) else GO(false)
#undef GO
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// Read-outs of the delta rule: q, k: activated rows [T, ld_in] (key head g at column g dim), u: [T, ld_u] (head h at column h vdim),
// p.s_hi / s_lo, prefix, fk: from delta_chunk.cu.
B200_API int b200_delta_out(const void* q, const void* k, const void* u, const ChunkParams* Pp, int ld_u, int T, int n_chunks, void* stream, int* err) {
  ChunkParams p = *Pp;
  if (!b200_memory_chunk_supported(p.dim, p.vdim, 0) || T <= 0 || n_chunks <= 0 || n_chunks > 65535 || p.H <= 0 || p.H > 65535 || p.group <= 0 || p.H % p.group ||
      ((p.ld_in | p.ld_out | p.ld_g | ld_u) & 7) || !p.prefix || !p.fk || !p.chunks) return -1;
  if ((reinterpret_cast<uintptr_t>(p.out) | reinterpret_cast<uintptr_t>(p.gate_out) | reinterpret_cast<uintptr_t>(p.norm_w)) & 15) return -1;
  p.dimp = p.dim;
  p.vpad = (p.vdim + 15) & ~15;
  p.vrows = p.vpad;
  p.pk = (p.dim + 63) / 64;
  p.pv = (p.vdim + 63) / 64;
  p.err = err;
  CUtensorMap tq, tk, tu, th, tl;
  const uint64_t planes = static_cast<uint64_t>(n_chunks) * p.H;
  int rc = make_tmap_planes(&tq, q, p.dim, T, p.H / p.group, p.ld_in, p.dim, MC_C);
  if (!rc) rc = make_tmap_planes(&tk, k, p.dim, T, p.H / p.group, p.ld_in, p.dim, MC_C);
  if (!rc) rc = make_tmap_planes(&tu, u, p.vdim, T, p.H, ld_u, p.vdim, MC_C);
  if (!rc) rc = make_tmap_planes(&th, p.s_hi, p.dim, p.vpad, planes, p.dimp, static_cast<uint64_t>(p.vpad) * p.dimp, p.vpad);
  if (!rc) rc = make_tmap_planes(&tl, p.s_lo, p.dim, p.vpad, planes, p.dimp, static_cast<uint64_t>(p.vpad) * p.dimp, p.vpad);
  if (rc) return rc;
  const int smem = mc_smem_out(p.pk, p.pv, p.vpad);
  int cols = 256;
  while (cols < MC_C + ((p.vpad + 31) & ~31)) cols <<= 1;
  const CUtensorMap tm[5] = {tq, tk, tu, th, tl};
  return dispatch_chunk_out<DELTA>(tm, p, n_chunks, smem, cols, reinterpret_cast<cudaStream_t>(stream));
}
