// Matrix memories with the gated delta rule, other than the tensor-core kernels of delta_chunk.cu:
//   * short_conv : causal convolution over the last tokens of every channel, then silu, for packed prompts; the newest inputs go to
//                  the sequence's ring
//   * delta_scan : token-by-token recurrence per (sequence, head), from the activated rows of a prompt or (RAW) the projection row of
//                  a decode step; unit norms, gates, state update, read-out, head norm and output gate
// S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q, formed as  a = S^T k, b = S^T q (one pass over the old state),
// u = beta (v - g a),  o = g b + (k . q) u.
// Storage types: bf16 (serving) or fp32; arithmetic is fp32.  This file is built without fast-math approximations.
#include "rowops.cuh"

namespace b200 {

// ------------------------------------------------------------------------------------------------ short convolution
constexpr int SC_CHUNK = 128, SC_PART = 64;         // tokens per chunk of the table, per CTA

struct ConvArgs {
  int ch, taps, ld_in, ld_out;                    // channels: a multiple of eight
  const float* w;                                 // [taps, ch], the last row meets the current token
  const int4* chunks;                             // {first token, tokens, sequence, -}
  const int4* seqs;                               // {first chunk, chunks, cache row, first position}
};

// Eight neighbouring elements as they lie in memory.
template <typename T> struct Raw8;
template <> struct Raw8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) { a = reinterpret_cast<const float4*>(p)[0]; b = reinterpret_cast<const float4*>(p)[1]; }
  __device__ __forceinline__ void get(float (&v)[8]) const { v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w; }
};
template <> struct Raw8<__nv_bfloat16> {
  uint4 q;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { q = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void get(float (&v)[8]) const {
    const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = unpack_bf16x2(w[j]);
      v[2 * j] = f.x;
      v[2 * j + 1] = f.y;
    }
  }
};

// 32 groups of eight channels x 8 runs of eight tokens, which are on their way at a time.  The CTA of a portion's first chunk is the only one that reads the ring, so it
// may write it afterwards.  TAPS: taps kept in registers (0: any number, inputs read again).
template <typename T, int TAPS>
__global__ void __launch_bounds__(256)
short_conv_kernel(const T* __restrict__ in, T* __restrict__ out, T* __restrict__ ring, const ConvArgs A) {
  const int c = (blockIdx.x * 32 + (threadIdx.x & 31)) * 8, ty = threadIdx.x >> 5;
  const int chunk = blockIdx.y / (SC_CHUNK / SC_PART), skip = blockIdx.y % (SC_CHUNK / SC_PART) * SC_PART;
  const int4 ck = A.chunks[chunk];
  const int4 sq = A.seqs[ck.z];
  const int t0 = ck.x + skip, n = min(SC_PART, ck.y - skip), i0 = (chunk - sq.x) * SC_CHUNK + skip;      // i0: index inside the portion
  if (n <= 0) return;
  const int taps = TAPS ? TAPS : A.taps;
  const bool live = c < A.ch;
  T* rg = ring + static_cast<size_t>(sq.z) * taps * A.ch + c;
  auto input = [&](int k, float (&v)[8]) {                      // input of token k of the chunk (k may be negative)
    const int p = sq.w + i0 + k;
    if (i0 + k >= 0) {
      ld8(in + static_cast<size_t>(t0 + k) * A.ld_in + c, v);
    } else if (p >= 0) {
      ld8(rg + static_cast<size_t>(p % taps) * A.ch, v);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] = 0.f;
    }
  };
  const int k0 = ty * 8, k1 = min(n, k0 + 8);
  if (live && k0 < k1) {
    if constexpr (TAPS > 0) {
      float w[TAPS][8], x[TAPS][8];                             // x[j]: input of j tokens ago
#pragma unroll
      for (int j = 0; j < TAPS; ++j) ld8(A.w + static_cast<size_t>(TAPS - 1 - j) * A.ch + c, w[j]);
      Raw8<T> raw[8];
#pragma unroll
      for (int k = 0; k < 8; ++k)
        if (k0 + k < k1) raw[k].load(in + static_cast<size_t>(t0 + k0 + k) * A.ld_in + c);
#pragma unroll
      for (int j = 1; j < TAPS; ++j) input(k0 - j, x[j - 1]);
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        if (k0 + k >= k1) break;
#pragma unroll
        for (int j = TAPS - 1; j > 0; --j)
#pragma unroll
          for (int e = 0; e < 8; ++e) x[j][e] = x[j - 1][e];
        raw[k].get(x[0]);
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          float s = 0.f;
#pragma unroll
          for (int j = 0; j < TAPS; ++j) s += w[j][e] * x[j][e];
          v[e] = sizeof(T) == 2 ? __fdividef(s, 1.f + __expf(-s)) : silu_f(s);
        }
        st8(out + static_cast<size_t>(t0 + k0 + k) * A.ld_out + c, v);
      }
    } else {
      for (int k = k0; k < k1; ++k) {
        float s[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        for (int j = 0; j < taps; ++j) {
          float w[8], x[8];
          ld8(A.w + static_cast<size_t>(taps - 1 - j) * A.ch + c, w);
          input(k - j, x);
#pragma unroll
          for (int e = 0; e < 8; ++e) s[e] += w[e] * x[e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) s[e] = silu_f(s[e]);
        st8(out + static_cast<size_t>(t0 + k) * A.ld_out + c, s);
      }
    }
  }
  if (i0 != 0) return;
  __syncthreads();                                              // the ring has been read
  if (!live) return;
  const int4 last = A.chunks[sq.x + sq.y - 1];
  const int len = last.x + last.y - t0;
  for (int r = ty; r < min(taps, len); r += 8) {
    const int i = len - 1 - r;
    float v[8];
    ld8(in + static_cast<size_t>(t0 + i) * A.ld_in + c, v);
    st8(rg + static_cast<size_t>((sq.w + i) % taps) * A.ch, v);
  }
}

// ------------------------------------------------------------------------------------------------ recurrence
struct DeltaArgs {
  int H, G, dim, vdim, ldv;       // ldv: row pitch of the state [rows, H, dim, ldv]
  int ld_in, off_q, off_k, off_v; // rows with q, k and v: activated, or (RAW) projections
  int ld_g, off_g, off_ba;        // projection rows: output gate; step size and decay (RAW)
  int ba_t, ba_h;                 // strides of `ba`
  int ld_out, ch, taps;
  float qscale, eps;
  const int4* seqs;               // {first token, tokens, cache row, first position}; null: one token per sequence at pos / row
  const int* pos;
  const int* row;
  const float* ba;                // [T, 2 H] projections of step size | decay (not RAW)
  const float *a_log, *dt_bias;   // [H]
  const float* norm_w;            // [vdim]
  const float* conv_w;            // [taps, ch]
  float* state;
};

__device__ __forceinline__ void cp_async16_zfill(uint32_t dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(on ? 16 : 0) : "memory");
}

// CTA per (head, sequence): warps over the key rows, float4 groups of value columns over the lanes.  R: float4 of the state per thread,
// held in registers or (RAW) in shared memory of its own, which leaves room for a third CTA; 0: the state stays in memory.
template <typename TI, typename T, bool RAW, int R>
__global__ void __launch_bounds__(256, R && !RAW ? 2 : 3)
delta_scan_kernel(const TI* __restrict__ in, const TI* __restrict__ gate, T* __restrict__ ring, T* __restrict__ out, const DeltaArgs M) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  const int h = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int t0 = blockIdx.y, n = 1, row, start;
  if (M.seqs) {
    const int4 s = M.seqs[blockIdx.y];
    t0 = s.x; n = s.y; row = s.z; start = s.w;
  } else {
    row = M.row[t0];
    start = M.pos[t0];
  }
  const int dim = M.dim, ldv = M.ldv, vdim = M.vdim, group = M.H / M.G, g = h / group, dp = (dim + 3) & ~3;
  float* qs = sm;                                  // [dim]
  float* ks = qs + dp;                             // [dim]
  float* vs = ks + dp;                             // [ldv]
  float* us = vs + ldv;                            // [ldv]
  float* part = us + ldv;                          // [2][8][ldv]
  float* red = part + 16 * ldv;                    // [32]
  float* gstate = M.state + (static_cast<size_t>(row) * M.H + h) * dim * ldv;
  int cl = 1;                                      // cl lanes of four columns, 32 / cl rows per warp
  while (4 * cl < ldv && cl < 32) cl <<= 1;
  const int rpw = 32 / cl, sub = lane / cl, col0 = 4 * (lane % cl), rstep = 8 * rpw, r0 = warp * rpw + sub;
  const int nu = (dim + rstep - 1) / rstep, nc = (ldv + 4 * cl - 1) / (4 * cl);      // row steps, column blocks
  const bool fresh = start == 0;
  constexpr bool STAGED = RAW && R > 0;
  float4 S[R && !STAGED ? R : 1];
  float4* own = reinterpret_cast<float4*>(red + 32) + tid;      // STAGED: piece e of this thread at 256 e
  if constexpr (STAGED) {
    int u = 0, cb = 0;
#pragma unroll
    for (int e = 0; e < R; ++e) {
      const int d = r0 + u * rstep, c = cb * 4 * cl + col0;
      const bool on = !fresh && cb < nc && d < dim && c < ldv;
      cp_async16_zfill(smem_u32(own + 256 * e), on ? gstate + static_cast<size_t>(d) * ldv + c : gstate, on);
      if (++u == nu) { u = 0; ++cb; }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  } else if constexpr (R > 0) {
    int u = 0, cb = 0;
#pragma unroll
    for (int e = 0; e < R; ++e) {
      const int d = r0 + u * rstep, c = cb * 4 * cl + col0;
      S[e] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && cb < nc && d < dim && c < ldv) S[e] = *reinterpret_cast<const float4*>(gstate + static_cast<size_t>(d) * ldv + c);
      if (++u == nu) { u = 0; ++cb; }
    }
  }
  const float decay_rate = -expf(M.a_log[h]), dt = M.dt_bias[h];
  for (int j = 0; j < n; ++j) {
    const size_t t = static_cast<size_t>(t0) + j;
    const TI* r = in + t * M.ld_in;
    __syncthreads();                               // the previous token's vectors have been read
    // channels [q | k | v]: activated already, or convolved here (a channel's ring gets its input from one CTA), two per thread at a time with
    // everything requested before anything is used
    const int total = 2 * dim + ldv;
    auto column = [&](int i) { return i < dim ? M.off_q + g * dim + i : i < 2 * dim ? M.off_k + g * dim + (i - dim) : M.off_v + h * vdim + (i - 2 * dim); };
    auto put = [&](int i, float v) { (i < dim ? qs + i : i < 2 * dim ? ks + (i - dim) : vs + (i - 2 * dim))[0] = v; };
    if constexpr (RAW) {
      constexpr int N = 4;                         // taps held at a time
      T* rg = ring + static_cast<size_t>(row) * M.taps * M.ch;
      const int now = start % M.taps;
      auto slot = [&](int back) { const int s = now - back; return static_cast<size_t>(s < 0 ? s + M.taps : s) * M.ch; };   // of `back` tokens ago
      for (int i0 = tid; i0 < total; i0 += 512) {
        float x[2][N], w[2][N];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = i0 + 256 * e, col = column(i);
          const bool on = i < total && i < 2 * dim + vdim;
#pragma unroll
          for (int b = 0; b < N; ++b) {
            const bool has = on && b < M.taps && b <= start;
            x[e][b] = !has ? 0.f : b == 0 ? ldf(r + col) : ldf(rg + slot(b) + col);
            w[e][b] = has ? M.conv_w[static_cast<size_t>(M.taps - 1 - b) * M.ch + col] : 0.f;
          }
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = i0 + 256 * e, col = column(i);
          if (i >= total) continue;
          float s = 0.f;
#pragma unroll
          for (int b = 0; b < N; ++b) s += w[e][b] * x[e][b];
          if (i < 2 * dim + vdim) {
            for (int b = N; b < M.taps && b <= start; ++b) s += M.conv_w[static_cast<size_t>(M.taps - 1 - b) * M.ch + col] * ldf(rg + slot(b) + col);
            if (i >= 2 * dim || h == g * group) stf(rg + slot(0) + col, x[e][0]);
          }
          put(i, silu_f(s));
        }
      }
    } else {
      for (int i = tid; i < total; i += 256) put(i, i < 2 * dim + vdim ? ldf(r + column(i)) : 0.f);
    }
    __syncthreads();
    float qq = 0.f, kk = 0.f, qk = 0.f;
    for (int i = tid; i < dim; i += 256) {
      const float q = qs[i], k = ks[i];
      qq += q * q;
      kk += k * k;
      qk += q * k;
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    qk = warp_sum(qk);
    if (lane == 0) { red[warp] = qq; red[8 + warp] = kk; red[16 + warp] = qk; }
    float zb, za;
    if constexpr (RAW) {
      zb = ldf(r + M.off_ba + h);
      za = ldf(r + M.off_ba + M.H + h);
    } else {
      zb = M.ba[t * M.ba_t + static_cast<size_t>(h) * M.ba_h];
      za = M.ba[t * M.ba_t + static_cast<size_t>(M.H + h) * M.ba_h];
    }
    const float beta = sigmoid_f(zb), gd = expf(decay_rate * softplus_f(za + dt));
    __syncthreads();
    qq = kk = qk = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) { qq += red[w]; kk += red[8 + w]; qk += red[16 + w]; }
    const float fq = M.qscale / sqrtf(qq + 1e-6f), fk = 1.f / sqrtf(kk + 1e-6f);
    const bool zero = fresh && j == 0;             // the stored state belongs to nobody
    // a = S^T k, b = S^T q
    auto flush = [&](int cb, float4 a, float4 b) {
      for (int o = 16; o >= cl; o >>= 1) {
        a.x += __shfl_xor_sync(0xffffffffu, a.x, o); a.y += __shfl_xor_sync(0xffffffffu, a.y, o);
        a.z += __shfl_xor_sync(0xffffffffu, a.z, o); a.w += __shfl_xor_sync(0xffffffffu, a.w, o);
        b.x += __shfl_xor_sync(0xffffffffu, b.x, o); b.y += __shfl_xor_sync(0xffffffffu, b.y, o);
        b.z += __shfl_xor_sync(0xffffffffu, b.z, o); b.w += __shfl_xor_sync(0xffffffffu, b.w, o);
      }
      const int c = cb * 4 * cl + col0;
      if (sub == 0 && c < ldv) {
        *reinterpret_cast<float4*>(part + warp * ldv + c) = a;
        *reinterpret_cast<float4*>(part + (8 + warp) * ldv + c) = b;
      }
    };
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
    auto gather = [&](const float4& s, int d) {
      const float k = ks[d], q = qs[d];
      a.x += k * s.x; a.y += k * s.y; a.z += k * s.z; a.w += k * s.w;
      b.x += q * s.x; b.y += q * s.y; b.z += q * s.z; b.w += q * s.w;
    };
    auto piece = [&](int e) -> float4 {
      if constexpr (STAGED) return own[256 * e];
      else return S[e];
    };
    if constexpr (R > 0) {
      if constexpr (STAGED) asm volatile("cp.async.wait_group 0;" ::: "memory");   // a thread reads what it has asked for itself
      int u = 0, cb = 0;
#pragma unroll
      for (int e = 0; e < R; ++e) {
        if (cb < nc) {
          const int d = r0 + u * rstep;
          if (d < dim) gather(piece(e), d);
          if (++u == nu) {
            flush(cb, a, b);
            a = b = make_float4(0.f, 0.f, 0.f, 0.f);
            u = 0;
            ++cb;
          }
        }
      }
    } else {
      for (int cb = 0; cb < nc; ++cb) {
        const int c = cb * 4 * cl + col0;
        a = b = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!zero && c < ldv)
          for (int d = r0; d < dim; d += rstep) gather(*reinterpret_cast<const float4*>(gstate + static_cast<size_t>(d) * ldv + c), d);
        __syncwarp();
        flush(cb, a, b);
      }
    }
    __syncthreads();
    float sq = 0.f;
    for (int c = tid; c < ldv; c += 256) {
      float sa = 0.f, sb = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) { sa += part[w * ldv + c]; sb += part[(8 + w) * ldv + c]; }
      const float u = beta * (vs[c] - gd * fk * sa), o = gd * fq * sb + qk * fq * fk * u;
      us[c] = fk * u;                              // with the raw k
      vs[c] = o;                                   // this thread reads it back below
      if (c < vdim) sq += o * o;
    }
    const float rms = 1.f / sqrtf(block_total<256>(sq, red) / static_cast<float>(vdim) + M.eps);   // orders the writes of us, too
    for (int c = tid; c < vdim; c += 256) {
      const float z = ldf(gate + t * M.ld_g + M.off_g + h * vdim + c);
      stf(out + t * M.ld_out + h * vdim + c, vs[c] * rms * M.norm_w[c] * silu_f(z));
    }
    auto update = [&](float4 s, int d, int c) {
      const float k = ks[d];
      const float4 u = *reinterpret_cast<const float4*>(us + c);
      s.x = gd * s.x + k * u.x; s.y = gd * s.y + k * u.y; s.z = gd * s.z + k * u.z; s.w = gd * s.w + k * u.w;
      return s;
    };
    if constexpr (R > 0) {
      int u = 0, cb = 0;
#pragma unroll
      for (int e = 0; e < R; ++e) {
        const int d = r0 + u * rstep, c = cb * 4 * cl + col0;
        if (cb < nc && d < dim && c < ldv) {
          const float4 next = update(piece(e), d, c);
          if constexpr (!STAGED) S[e] = next;
          if (j + 1 == n) *reinterpret_cast<float4*>(gstate + static_cast<size_t>(d) * ldv + c) = next;
        }
        if (++u == nu) { u = 0; ++cb; }
      }
    } else {
      for (int cb = 0; cb < nc; ++cb) {
        const int c = cb * 4 * cl + col0;
        if (c < ldv)
          for (int d = r0; d < dim; d += rstep) {
            float4* p = reinterpret_cast<float4*>(gstate + static_cast<size_t>(d) * ldv + c);
            *p = update(zero ? make_float4(0.f, 0.f, 0.f, 0.f) : *p, d, c);
          }
      }
    }
  }
}

}  // namespace b200

using namespace b200;
typedef __nv_bfloat16 bf16_t;
#define STREAM reinterpret_cast<cudaStream_t>(stream)
#define DONE (cudaGetLastError() == cudaSuccess ? 0 : -2)

// in: projection rows, out: activated rows, ring: [rows, taps, ch]; all of one storage type.
B200_API int b200_short_conv(const void* in, void* out, void* ring, const ConvArgs* Ap, int n_chunks, int f32, void* stream) {
  const ConvArgs A = *Ap;
  if (n_chunks <= 0 || n_chunks > 32767 || A.ch <= 0 || ((A.ch | A.ld_in | A.ld_out) & 7) || A.taps < 1 || A.taps > SC_PART || !A.w || !A.chunks || !A.seqs ||
      ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(ring) | reinterpret_cast<uintptr_t>(A.w)) & 15)) return -1;
  const dim3 grid((A.ch / 8 + 31) / 32, n_chunks * (SC_CHUNK / SC_PART));
#define GO2(T_, N) short_conv_kernel<T_, N><<<grid, 256, 0, STREAM>>>((const T_*)in, (T_*)out, (T_*)ring, A)
#define GO(T_)                        \
  switch (A.taps) {                   \
    case 2: GO2(T_, 2); break;        \
    case 3: GO2(T_, 3); break;        \
    case 4: GO2(T_, 4); break;        \
    default: GO2(T_, 0);              \
  }
  if (f32) GO(float) else GO(bf16_t)
#undef GO
#undef GO2
  return DONE;
}

// raw: `in` are the projection rows of one token per sequence (fp32 with in_f32); otherwise activated rows of one storage type.
// gate: projection rows of the type of `in`.  n: sequences.
B200_API int b200_delta_scan(const void* in, const void* gate, void* ring, void* out, const DeltaArgs* Mp, int n, int raw, int in_f32, int f32,
                             void* stream) {
  const DeltaArgs M = *Mp;
  if (n <= 0 || n > 65535 || M.H <= 0 || M.G <= 0 || M.H % M.G || M.dim <= 0 || M.vdim <= 0 || M.ldv < M.vdim || (M.ldv & 3) || !M.state || !M.a_log || !M.dt_bias ||
      !M.norm_w || (f32 && !in_f32) || (!raw && in_f32 != f32) || (raw ? (!ring || !M.conv_w || M.taps < 1 || M.seqs) : !M.ba) || (!M.seqs && (!M.pos || !M.row))) return -1;
  const size_t smem = (2 * ((M.dim + 3) & ~3) + 18 * M.ldv + 32) * sizeof(float);
  if (smem > 220 * 1024) return -1;
  int cl = 1;
  while (4 * cl < M.ldv && cl < 32) cl <<= 1;
  const int rstep = 8 * (32 / cl), held = ((M.dim + rstep - 1) / rstep) * ((M.ldv + 4 * cl - 1) / (4 * cl));
#define GO2(TI, T_, RAW, R)                                                                                            \
  {                                                                                                                    \
    const size_t bytes = smem + (RAW ? R * 4096 : 0);                                                                   \
    if (bytes > 220 * 1024) return -1;                                                                                  \
    if (bytes > 48 * 1024 && cudaFuncSetAttribute(delta_scan_kernel<TI, T_, RAW, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                                  static_cast<int>(bytes)) != cudaSuccess) return -3;                   \
    launch_k(delta_scan_kernel<TI, T_, RAW, R>, dim3(M.H, n), dim3(256), bytes, STREAM, (const TI*)in, (const TI*)gate, (T_*)ring, (T_*)out, M); \
  }
#define GO(TI, T_, RAW) { if (held <= 4) GO2(TI, T_, RAW, 4) else if (held <= 16) GO2(TI, T_, RAW, 16) else GO2(TI, T_, RAW, 0) }
  if (raw) {
    if (f32) GO(float, float, true)
    else if (in_f32) GO(float, bf16_t, true)
    else GO(bf16_t, bf16_t, true)
  } else {
    if (f32) GO(float, float, false)
    else GO(bf16_t, bf16_t, false)
  }
#undef GO
#undef GO2
  return DONE;
}
