// Kernels of the layered decoder models that mix attention with recurrent memories, other than the tensor-core ones:
//   * sandwich_norm     : x += norm(a + bias) [+ step vector] on the fp32 residual stream, then the norm that feeds the next
//                         sublayer; layer norms, or RMS norms whose weights are stored around zero
//   * layernorm_rows    : gathered rows of the final norm
//   * glu               : act(gate) * up of a [gate | up] row, tanh-GELU or silu
//   * kv_append         : keys and values of a step into the cache
//   * memory_scan       : token-by-token recurrence of a matrix memory per (sequence, head): decode steps (one pass over the
//                         state) and any prompt (state in shared memory); fixed decay, or exponential gates with normaliser
//                         and running maximum
//   * memory_merge      : key splits of the decode attention with the heads' gates, and the norm over all heads of a decaying
//                         memory with its output gate
// Storage types: bf16 (serving) or fp32; arithmetic is fp32.  This file is built without fast-math approximations.
#include "rowops.cuh"

namespace b200 {

// ------------------------------------------------------------------------------------------------ layer norms
struct SandwichArgs {
  int E, ld_a, ld_h, clear, nzero;
  float eps, bias_mult, out_mult; // out_mult: factor on the next sublayer's input
  const float* bias;              // on the sublayer output, times bias_mult; null: none
  const float *w1, *b1;           // norm of the sublayer output
  const float* step;              // added to the stream afterwards; null: none
  const float *w2, *b2;           // norm of the next sublayer's input; null: none
  float* x;
  float* zero;                    // second accumulator, re-armed here
  // sublayer output that is still a sum (`a` holds the fp32 rows it picks from): sum_k weight[row, k] a[slot[row, k]], with mix_h[row] in
  // place of a row whose slot is negative, + weight[row, top] shared[row]
  int top, ld_mix, ld_shared;     // top 0: `a` is the output itself
  const int* slot;
  const float* weight;            // [rows, top + 1]
  const void *mix_h, *shared;     // operand precision; the type of `a` (null: none)
};

// One CTA per row; NV groups of eight columns per thread held in registers.  A null `a` skips the sublayer output.
// RMS: no means are taken, weights are one plus the stored ones and there are no biases.  SUM: the output is still a sum.
template <typename TI, typename T, int NV, bool RMS, bool SUM>
__global__ void __launch_bounds__(256)
sandwich_vec_kernel(TI* __restrict__ a, T* __restrict__ h, const SandwichArgs A) {
  pdl_trigger();
  if (gridDim.x <= 256) {                          // few rows: the weights' way from memory would add to the reductions'
    for (int i = 32 * threadIdx.x; i < A.E; i += 8192) {
      if (a) prefetch_l2(A.w1 + i);
      if (A.w2) prefetch_l2(A.w2 + i);
      if (!RMS && a) prefetch_l2(A.b1 + i);
      if (!RMS && A.w2) prefetch_l2(A.b2 + i);
    }
  }
  pdl_wait();
  __shared__ float red[8];
  const size_t row = blockIdx.x;
  const int nvec = A.E >> 3;
  const float invE = 1.f / static_cast<float>(A.E);
  float s[NV][8], xv[NV][8];
  float sum = 0.f;
  TI* ar = a ? a + row * A.ld_a : nullptr;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i < nvec) {
      ld8(A.x + row * A.E + 8 * i, xv[k]);
      if (ar) {
        if constexpr (SUM) sublayer_cols<8, TI, T>(A, a, row, 8 * i, s[k]);
        else ld8(ar + 8 * i, s[k]);
        if (A.clear) clear8(ar + 8 * i);
        if (A.bias) {
          float b[8];
          ld8(A.bias + 8 * i, b);
#pragma unroll
          for (int j = 0; j < 8; ++j) s[k][j] += A.bias_mult * b[j];
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) sum += s[k][j];
      }
    }
  }
  for (int i = threadIdx.x; i < A.nzero; i += 256) A.zero[row * A.nzero + i] = 0.f;
  if (ar) {
    const float mean = RMS ? 0.f : block_total<256>(sum, red) * invE;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k)
      if (threadIdx.x + k * 256 < nvec)
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          s[k][j] -= mean;
          ss += s[k][j] * s[k][j];
        }
    const float r = 1.f / sqrtf(block_total<256>(ss, red) * invE + A.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = threadIdx.x + k * 256;
      if (i < nvec) {
        float wv[8], bv[8];
        ld8(A.w1 + 8 * i, wv);
        if (!RMS) ld8(A.b1 + 8 * i, bv);
#pragma unroll
        for (int j = 0; j < 8; ++j) xv[k][j] += RMS ? s[k][j] * r * (1.f + wv[j]) : s[k][j] * r * wv[j] + bv[j];
      }
    }
  }
  sum = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i < nvec) {
      if (A.step) {
        float v[8];
        ld8(A.step + 8 * i, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) xv[k][j] += v[j];
      }
      if (ar || A.step) st8(A.x + row * A.E + 8 * i, xv[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) sum += xv[k][j];
    }
  }
  if (!A.w2) return;
  const float mean = RMS ? 0.f : block_total<256>(sum, red) * invE;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k)
    if (threadIdx.x + k * 256 < nvec)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        xv[k][j] -= mean;
        ss += xv[k][j] * xv[k][j];
      }
  const float r = 1.f / sqrtf(block_total<256>(ss, red) * invE + A.eps);
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i < nvec) {
      float wv[8], bv[8];
      ld8(A.w2 + 8 * i, wv);
      if (!RMS) ld8(A.b2 + 8 * i, bv);
#pragma unroll
      for (int j = 0; j < 8; ++j) xv[k][j] = (RMS ? xv[k][j] * r * (1.f + wv[j]) : xv[k][j] * r * wv[j] + bv[j]) * A.out_mult;
      st8(h + row * A.ld_h + 8 * i, xv[k]);
    }
  }
}

// Any width: several passes over the row.
template <typename TI, typename T, bool RMS, bool SUM>
__global__ void __launch_bounds__(256)
sandwich_kernel(TI* __restrict__ a, T* __restrict__ h, const SandwichArgs A) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const size_t row = blockIdx.x;
  const float invE = 1.f / static_cast<float>(A.E);
  TI* ar = a ? a + row * A.ld_a : nullptr;
  float* x = A.x + row * A.E;
  for (int i = threadIdx.x; i < A.nzero; i += 256) A.zero[row * A.nzero + i] = 0.f;
  auto in = [&](int i) {
    float v;
    if constexpr (SUM) sublayer_cols<1, TI, T>(A, a, row, i, &v);
    else v = ldf(ar + i);
    return v + (A.bias ? A.bias_mult * A.bias[i] : 0.f);
  };
  float mean = 0.f, r = 0.f;
  if (ar) {
    float sum = 0.f, ss = 0.f;
    for (int i = threadIdx.x; i < A.E; i += 256) sum += in(i);
    mean = RMS ? 0.f : block_total<256>(sum, red) * invE;
    for (int i = threadIdx.x; i < A.E; i += 256) {
      const float d = in(i) - mean;
      ss += d * d;
    }
    r = 1.f / sqrtf(block_total<256>(ss, red) * invE + A.eps);
  }
  float sum = 0.f, ss = 0.f;
  for (int i = threadIdx.x; i < A.E; i += 256) {
    float v = x[i];
    if (ar) {
      v += RMS ? in(i) * r * (1.f + A.w1[i]) : (in(i) - mean) * r * A.w1[i] + A.b1[i];
      if (A.clear) stf(ar + i, 0.f);
    }
    if (A.step) v += A.step[i];
    if (ar || A.step) x[i] = v;
    sum += v;
  }
  if (!A.w2) return;
  mean = RMS ? 0.f : block_total<256>(sum, red) * invE;
  for (int i = threadIdx.x; i < A.E; i += 256) {
    const float d = x[i] - mean;
    ss += d * d;
  }
  r = 1.f / sqrtf(block_total<256>(ss, red) * invE + A.eps);
  for (int i = threadIdx.x; i < A.E; i += 256)
    stf(h + row * A.ld_h + i, (RMS ? x[i] * r * (1.f + A.w2[i]) : (x[i] - mean) * r * A.w2[i] + A.b2[i]) * A.out_mult);
}

template <typename T>
__global__ void __launch_bounds__(256)
layernorm_rows_kernel(const float* __restrict__ x, const int* __restrict__ idx, const float* __restrict__ w, const float* __restrict__ b,
                      T* __restrict__ y, int ld_y, int E, float eps) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const float* xr = x + static_cast<size_t>(idx ? idx[blockIdx.x] : static_cast<int>(blockIdx.x)) * E;
  const float invE = 1.f / static_cast<float>(E);
  float sum = 0.f, ss = 0.f;
  for (int i = threadIdx.x; i < E; i += 256) sum += xr[i];
  const float mean = block_total<256>(sum, red) * invE;
  for (int i = threadIdx.x; i < E; i += 256) ss += (xr[i] - mean) * (xr[i] - mean);
  const float r = 1.f / sqrtf(block_total<256>(ss, red) * invE + eps);
  for (int i = threadIdx.x; i < E; i += 256) stf(y + static_cast<size_t>(blockIdx.x) * ld_y + i, (xr[i] - mean) * r * w[i] + b[i]);
}

// ------------------------------------------------------------------------------------------------ gated feed-forward
// y = act(gate) * up of rows [gate (N) | up (N)]; act: gelu (tanh form) or silu
template <typename TI, typename T, bool SILU>
__global__ void __launch_bounds__(256)
glu_kernel(TI* __restrict__ a, int ld_a, int clear, T* __restrict__ y, int ld_y, int N) {
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.y;
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i >= N) return;
  TI* p = a + row * ld_a + i;
  const float g = ldf(p), u = ldf(p + N);
  if (clear) {
    stf(p, 0.f);
    stf(p + N, 0.f);
  }
  stf(y + row * ld_y + i, (SILU ? silu_f(g) : 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)))) * u);
}

// ------------------------------------------------------------------------------------------------ keys and values
// cache[row[t], pos[t], 0 .. width) = in[t, 0 .. width) (+ bias): the projections of k and v lie side by side in both.
template <typename TI, typename T>
__global__ void __launch_bounds__(256)
kv_append_kernel(const TI* __restrict__ in, int ld_in, const float* __restrict__ bias, T* __restrict__ cache, int width, int ld_kv,
                 int cap, const int* __restrict__ pos, const int* __restrict__ row, int total) {
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x * 256 + threadIdx.x;              // eight elements each; rows and widths are multiples of eight
  if (i >= total) return;
  const int per = width >> 3, t = i / per, c = 8 * (i - t * per);
  float v[8];
  ld8(in + static_cast<size_t>(t) * ld_in + c, v);
  if (bias) {
    float b[8];
    ld8(bias + c, b);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] += b[j];
  }
  st8(cache + (static_cast<size_t>(row[t]) * cap + pos[t]) * ld_kv + c, v);
}

// ------------------------------------------------------------------------------------------------ matrix memories
struct MemoryArgs {
  int H, dim, vdim, ldv;          // ldv: row pitch of the state [rows, H, dim, ldv]
  int ld_in, off_q, off_k, off_v, off_g;
  int ld_out, E, ld_h, ld_w, gate_t, gate_h;   // gate_t, gate_h: strides of `gates` per token and per gate
  int silu;                       // q, k and v are raw projections: apply silu
  int stage;                      // keep the state in shared memory between tokens
  float qscale, cap, eps;
  const int4* seqs;               // {first token, tokens, cache row, first position}; null: one token per sequence at pos / row
  const int* pos;
  const int* row;
  const float* decay;             // fixed decay per head; null: gated
  const float* gates;             // [T, 2H] (strided) raw log input | log forget gate projections; null: formed here from h and w_gate
  const float* gate_bias;         // [2H]
  float* state;
  float* stab;                    // [rows, H, dim + 1]: normaliser, running maximum
  const float* norm_w;            // gated: [H * vdim]
  float* out32;                   // decay: [T, ld_out] fp32
};

// CTA per (head, sequence): warps over the key rows, float4 groups of value columns over the lanes.  Fixed decay: out32 gets
// S^T q.  Gated: the head's output is normalised, RMS-normed, gated and stored in `out`.
template <typename TI, typename T, bool GATED>
__global__ void __launch_bounds__(256, 3)
memory_scan_kernel(const TI* __restrict__ in, const T* __restrict__ hin, const T* __restrict__ w_gate, T* __restrict__ out, const MemoryArgs M) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];
  const int h = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int t0 = blockIdx.y, n = 1, row, start;
  if (M.seqs) {
    const int4 s = M.seqs[blockIdx.y];
    t0 = s.x; n = s.y; row = s.z; start = s.w;
  } else {
    row = M.row[t0];
    start = M.pos[t0];
  }
  const int dim = M.dim, ldv = M.ldv, vdim = M.vdim;
  float* qs = sm;                                  // [dim]
  float* ks = qs + ((dim + 3) & ~3);               // [dim]
  float* vs = ks + ((dim + 3) & ~3);               // [ldv]
  float* part = vs + ldv;                          // [8][ldv]
  float* red = part + 8 * ldv;                     // [16]
  float* ns = red + 16;                            // [dim]
  float* ss = ns + ((dim + 3) & ~3);               // [dim][ldv] with `stage`
  float* gstate = M.state + (static_cast<size_t>(row) * M.H + h) * dim * ldv;
  if (!M.seqs && start > 0)                        // the state is on its way while the token's vectors and gates are formed
    for (int i = 32 * tid; i < dim * ldv; i += 8192) prefetch_l2(gstate + i);
  float* gstab = GATED ? M.stab + (static_cast<size_t>(row) * M.H + h) * (dim + 1) : nullptr;
  // lanes over columns: cl lanes of four columns, 32 / cl rows per warp
  int cl = 1;
  while (4 * cl < ldv && cl < 32) cl <<= 1;
  const int rpw = 32 / cl, sub = lane / cl, col0 = 4 * (lane % cl), rstep = 8 * rpw, r0 = warp * rpw + sub;
  const bool fresh = start == 0;
  float* S = M.stage ? ss : gstate;
  if (M.stage) {
    for (int i = tid; i < dim * ldv / 4; i += 256)
      reinterpret_cast<float4*>(ss)[i] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : reinterpret_cast<const float4*>(gstate)[i];
  }
  float m = 0.f;
  if constexpr (GATED) {
    for (int i = tid; i < dim; i += 256) ns[i] = fresh ? 0.f : gstab[i];
    m = fresh ? 0.f : gstab[dim];
  }
  const float fixed = GATED ? 0.f : M.decay[h];
  for (int j = 0; j < n; ++j) {
    const size_t t = static_cast<size_t>(t0) + j;
    const TI* r = in + t * M.ld_in;
    __syncthreads();                               // the previous token's vectors and partial sums have been read
    for (int i = tid; i < dim; i += 256) {
      float q = ldf(r + M.off_q + h * dim + i), k = ldf(r + M.off_k + h * dim + i);
      if (M.silu) { q = silu_f(q); k = silu_f(k); }
      qs[i] = q * M.qscale;
      ks[i] = k;
    }
    for (int i = tid; i < ldv; i += 256) {
      float v = i < vdim ? ldf(r + M.off_v + h * vdim + i) : 0.f;
      if (M.silu) v = silu_f(v);
      vs[i] = v;
    }
    float a = fixed, b = 1.f;
    if constexpr (GATED) {
      float zi, zf;
      if (M.gates) {
        zi = M.gates[t * M.gate_t + static_cast<size_t>(h) * M.gate_h];
        zf = M.gates[t * M.gate_t + static_cast<size_t>(M.H + h) * M.gate_h];
      } else {
        const T* x = hin + t * M.ld_h;
        const T* wi = w_gate + static_cast<size_t>(h) * M.ld_w;
        const T* wf = w_gate + static_cast<size_t>(M.H + h) * M.ld_w;
        float si = 0.f, sf = 0.f;
        for (int i = tid; i < M.E; i += 256) {
          const float xv = ldf(x + i);
          si += xv * ldf(wi + i);
          sf += xv * ldf(wf + i);
        }
        si = warp_sum(si);
        sf = warp_sum(sf);
        if (lane == 0) { red[warp] = si; red[8 + warp] = sf; }
        __syncthreads();
        zi = zf = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) { zi += red[w]; zf += red[8 + w]; }
      }
      zi += M.gate_bias[h];
      zf += M.gate_bias[M.H + h];
      const float li = M.cap * tanhf(zi / M.cap), z = M.cap * tanhf(zf / M.cap);
      const float lf = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));      // log sigmoid
      const float mn = fmaxf(lf + m, li);
      a = expf(lf + m - mn);
      b = expf(li - mn);
      m = mn;
    }
    __syncthreads();
    float nq = 0.f;
    if constexpr (GATED) {
      for (int i = tid; i < dim; i += 256) {
        const float v = a * ns[i] + b * ks[i];
        ns[i] = v;
        nq += v * qs[i];
      }
    }
    const bool zero = fresh && j == 0;             // the stored state belongs to nobody
    for (int c0 = 0; c0 < ldv; c0 += 4 * cl) {      // uniform over the warp
      const int c = c0 + col0, dend = c < ldv ? dim : 0;
      const float4 v = c < ldv ? *reinterpret_cast<const float4*>(vs + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 bv = make_float4(b * v.x, b * v.y, b * v.z, b * v.w);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
      constexpr int U = 8;                         // state rows in flight per thread
      for (int d0 = r0; d0 < dend; d0 += U * rstep) {
        float4 s[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int d = d0 + u * rstep;
          s[u] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (d < dim && !zero) s[u] = *reinterpret_cast<const float4*>(S + static_cast<size_t>(d) * ldv + c);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int d = d0 + u * rstep;
          if (d < dim) {
            const float k = ks[d], q = qs[d];
            s[u].x = a * s[u].x + k * bv.x; s[u].y = a * s[u].y + k * bv.y;
            s[u].z = a * s[u].z + k * bv.z; s[u].w = a * s[u].w + k * bv.w;
            *reinterpret_cast<float4*>(S + static_cast<size_t>(d) * ldv + c) = s[u];
            o.x += q * s[u].x; o.y += q * s[u].y; o.z += q * s[u].z; o.w += q * s[u].w;
          }
        }
      }
      for (int off = 16; off >= cl; off >>= 1) {
        o.x += __shfl_xor_sync(0xffffffffu, o.x, off); o.y += __shfl_xor_sync(0xffffffffu, o.y, off);
        o.z += __shfl_xor_sync(0xffffffffu, o.z, off); o.w += __shfl_xor_sync(0xffffffffu, o.w, off);
      }
      if (sub == 0 && c < ldv) *reinterpret_cast<float4*>(part + warp * ldv + c) = o;
    }
    if constexpr (GATED) {
      nq = warp_sum(nq);
      if (lane == 0) red[warp] = nq;
    }
    __syncthreads();
    if constexpr (!GATED) {
      for (int c = tid; c < vdim; c += 256) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) o += part[w * ldv + c];
        M.out32[t * M.ld_out + h * vdim + c] = o;
      }
    } else {
      float d = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) d += red[w];
      const float inv = 1.f / (fmaxf(fabsf(d), expf(-m)) + 1e-6f);
      float sq = 0.f;
      for (int c = tid; c < vdim; c += 256) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) o += part[w * ldv + c];
        o *= inv;
        vs[c] = o;                                 // this thread reads it back below
        sq += o * o;
      }
      const float rms = 1.f / sqrtf(block_total<256>(sq, red) / static_cast<float>(vdim) + M.eps);
      for (int c = tid; c < vdim; c += 256) {
        const float g = sigmoid_f(ldf(r + M.off_g + h * vdim + c));
        stf(out + t * M.ld_out + h * vdim + c, vs[c] * rms * M.norm_w[h * vdim + c] * g);
      }
    }
  }
  __syncthreads();
  if (M.stage)
    for (int i = tid; i < dim * ldv / 4; i += 256) reinterpret_cast<float4*>(gstate)[i] = reinterpret_cast<const float4*>(ss)[i];
  if constexpr (GATED) {
    for (int i = tid; i < dim; i += 256) gstab[i] = ns[i];
    if (tid == 0) gstab[dim] = m;
  }
}

// ------------------------------------------------------------------------------------------------ joining the halves
struct MergeArgs {
  int H, vdim, splits, HR, rvdim;
  int ld_in, off_lg, off_rg;      // gates in the projection row: one per attention head, one per memory output
  int ld_mem, ld_out, off_r;      // memory outputs start at column off_r
  float left_scale, right_scale, eps;
  const float* part_o;            // [T, H, splits, vdim padded to eight]; H = 0: the attention part is in place already
  const float* part_ml;
  const float* norm_w;            // [HR * rvdim]
};

// CTA (token, slice): slice 0 the norm over all memory heads with its gate, the others eight attention heads each.
template <typename TI, typename TM, typename T>
__global__ void __launch_bounds__(256)
memory_merge_kernel(const TI* __restrict__ in, const TM* __restrict__ mem, T* __restrict__ out, const MergeArgs A) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const size_t t = blockIdx.x;
  const TI* r = in + t * A.ld_in;
  if (blockIdx.y == 0) {
    const int W = A.HR * A.rvdim;
    const TM* m = mem + t * A.ld_mem;
    const TI* g = r + A.off_rg;
    T* o = out + t * A.ld_out + A.off_r;
    constexpr int KEEP = 8;                        // float4 groups per thread held over the norm
    if ((W & 3) == 0 && W <= 1024 * KEEP) {
      float v[KEEP][4];
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = 4 * (threadIdx.x + 256 * k);
        if (i < W) {
          ld4(m + i, v[k]);
#pragma unroll
          for (int j = 0; j < 4; ++j) ss += v[k][j] * v[k][j];
        }
      }
      const float rms = A.right_scale / sqrtf(block_total<256>(ss, red) / static_cast<float>(W) + A.eps);
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int i = 4 * (threadIdx.x + 256 * k);
        if (i < W) {
          float gv[4], wv[4];
          ld4(g + i, gv);
          ld4(A.norm_w + i, wv);
#pragma unroll
          for (int j = 0; j < 4; ++j) v[k][j] *= rms * wv[j] * sigmoid_f(gv[j]);
          st2(o + i, make_float2(v[k][0], v[k][1]));
          st2(o + i + 2, make_float2(v[k][2], v[k][3]));
        }
      }
      return;
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < W; i += 256) {
      const float v = ldf(m + i);
      ss += v * v;
    }
    const float rms = A.right_scale / sqrtf(block_total<256>(ss, red) / static_cast<float>(W) + A.eps);
    for (int i = threadIdx.x; i < W; i += 256) stf(o + i, ldf(m + i) * rms * A.norm_w[i] * sigmoid_f(ldf(g + i)));
    return;
  }
  const int h = (blockIdx.y - 1) * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= A.H) return;
  const size_t base = (t * A.H + h) * A.splits;
  const float2 e = lane < A.splits ? *reinterpret_cast<const float2*>(A.part_ml + (base + lane) * 2) : make_float2(-INFINITY, 0.f);
  const float mm = warp_max(e.x);
  const float a = e.x == -INFINITY ? 0.f : expf(e.x - mm);
  const float mine = a / warp_sum(a * e.y) * sigmoid_f(ldf(r + A.off_lg + h)) * A.left_scale;
  const int vs = (A.vdim + 7) & ~7;
  const float* p = A.part_o + base * vs;
  for (int c = 4 * lane; c - 4 * lane < A.vdim; c += 128) {   // uniform over the warp
    float o[4] = {0.f, 0.f, 0.f, 0.f};
    constexpr int U = 8;                             // split rows in flight
    for (int s0 = 0; s0 < A.splits; s0 += U) {
      float x[U][4];
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (s0 + u < A.splits && c < vs) ld4(p + static_cast<size_t>(s0 + u) * vs + c, x[u]);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const float w = __shfl_sync(0xffffffffu, mine, (s0 + u) & 31);
        if (s0 + u < A.splits && c < vs && w != 0.f) {   // an empty split's partial is not initialised
#pragma unroll
          for (int k = 0; k < 4; ++k) o[k] += w * x[u][k];
        }
      }
    }
    T* dst = out + t * A.ld_out + h * A.vdim + c;
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (c + k < A.vdim) stf(dst + k, o[k]);
  }
}

// The memory half alone, for prompts (bf16): a warp per token, all of a row's pieces requested at once.  W = HR * rvdim, a
// multiple of eight up to 256 * G.
template <int G>
__global__ void __launch_bounds__(128)
memory_norm_rows_kernel(const __nv_bfloat16* __restrict__ in, const __nv_bfloat16* __restrict__ mem, __nv_bfloat16* __restrict__ out,
                        const MergeArgs A, int rows) {
  const size_t t = static_cast<size_t>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  if (t >= rows) return;
  const int lane = threadIdx.x & 31, W = A.HR * A.rvdim;
  const __nv_bfloat16* m = mem + t * A.ld_mem;
  const __nv_bfloat16* g = in + t * A.ld_in + A.off_rg;
  __nv_bfloat16* o = out + t * A.ld_out + A.off_r;
  uint4 v[G], q[G];
#pragma unroll
  for (int k = 0; k < G; ++k) {
    const int i = 8 * (lane + 32 * k);
    v[k] = make_uint4(0u, 0u, 0u, 0u);
    if (i < W) {
      v[k] = *reinterpret_cast<const uint4*>(m + i);
      q[k] = *reinterpret_cast<const uint4*>(g + i);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < G; ++k) {
    const uint32_t w[4] = {v[k].x, v[k].y, v[k].z, v[k].w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = unpack_bf16x2(w[j]);
      ss += f.x * f.x + f.y * f.y;
    }
  }
  const float rms = A.right_scale / sqrtf(warp_sum(ss) / static_cast<float>(W) + A.eps);
#pragma unroll
  for (int k = 0; k < G; ++k) {
    const int i = 8 * (lane + 32 * k);
    if (i < W) {
      const uint32_t vw[4] = {v[k].x, v[k].y, v[k].z, v[k].w}, gw[4] = {q[k].x, q[k].y, q[k].z, q[k].w};
      float wv[8], r[8];
      ld8(A.norm_w + i, wv);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 x = unpack_bf16x2(vw[j]), z = unpack_bf16x2(gw[j]);
        r[2 * j] = x.x * rms * wv[2 * j] * __fdividef(1.f, 1.f + __expf(-z.x));
        r[2 * j + 1] = x.y * rms * wv[2 * j + 1] * __fdividef(1.f, 1.f + __expf(-z.y));
      }
      st8(o + i, r);
    }
  }
}

}  // namespace b200

using namespace b200;
typedef __nv_bfloat16 bf16_t;
#define STREAM reinterpret_cast<cudaStream_t>(stream)
#define DONE (cudaGetLastError() == cudaSuccess ? 0 : -2)

// Every `f32` argument: the operand storage type is fp32 instead of bf16; `in_f32`: the GEMM output is fp32.

template <typename TI, typename T, bool RMS, bool SUM = false>
static void launch_sandwich(void* a, void* h, const SandwichArgs& A, int rows, cudaStream_t st) {
  const bool vec = A.E % 8 == 0 && A.ld_a % 8 == 0 && A.ld_h % 8 == 0 && A.ld_mix % 8 == 0 && A.ld_shared % 8 == 0 &&
                   !((reinterpret_cast<uintptr_t>(A.mix_h) | reinterpret_cast<uintptr_t>(A.shared)) & 15) &&
                   !((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(A.x) |
                      reinterpret_cast<uintptr_t>(A.w1) | reinterpret_cast<uintptr_t>(A.b1) | reinterpret_cast<uintptr_t>(A.w2) |
                      reinterpret_cast<uintptr_t>(A.b2) | reinterpret_cast<uintptr_t>(A.bias) | reinterpret_cast<uintptr_t>(A.step)) & 15);
  const int nv = vec ? (A.E / 8 + 255) / 256 : 0;
#define GO(NV) launch_k(sandwich_vec_kernel<TI, T, NV, RMS, SUM>, dim3(rows), dim3(256), 0, st, (TI*)a, (T*)h, A)
  if (nv == 1) GO(1);
  else if (nv == 2) GO(2);
  else if (nv == 3) GO(3);
  else if (nv == 4) GO(4);
  else launch_k(sandwich_kernel<TI, T, RMS, SUM>, dim3(rows), dim3(256), 0, st, (TI*)a, (T*)h, A);
#undef GO
}

// rms: RMS norms, weights stored around zero, no biases
B200_API int b200_sandwich_norm(void* a, void* h, const SandwichArgs* Ap, int rows, int in_f32, int f32, int rms, void* stream) {
  const SandwichArgs A = *Ap;
  if (rows <= 0 || A.E <= 0 || !A.x || (A.clear && !in_f32) || (f32 && !in_f32) || (A.nzero && !A.zero)) return -1;
  if (A.top && (!rms || !in_f32 || !a || A.top < 0 || A.clear || !A.slot || !A.weight || !A.mix_h)) return -1;
  if ((a && (!A.w1 || (!rms && !A.b1))) || (A.w2 && ((!rms && !A.b2) || !h))) return -1;
#define GO(RMS)                                                                \
  {                                                                            \
    if (f32) launch_sandwich<float, float, RMS>(a, h, A, rows, STREAM);        \
    else if (in_f32) launch_sandwich<float, bf16_t, RMS>(a, h, A, rows, STREAM); \
    else launch_sandwich<bf16_t, bf16_t, RMS>(a, h, A, rows, STREAM);          \
  }
  if (A.top) {                       // few rows: the experts' are fp32
    if (f32) launch_sandwich<float, float, true, true>(a, h, A, rows, STREAM);
    else launch_sandwich<float, bf16_t, true, true>(a, h, A, rows, STREAM);
  } else if (rms) GO(true) else GO(false)
#undef GO
  return DONE;
}

B200_API int b200_layernorm_rows(const float* x, const int* idx, const float* w, const float* b, void* y, int ld_y, int rows, int E,
                                 float eps, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (f32) launch_k(layernorm_rows_kernel<float>, dim3(rows), dim3(256), 0, STREAM, x, idx, w, b, (float*)y, ld_y, E, eps);
  else launch_k(layernorm_rows_kernel<bf16_t>, dim3(rows), dim3(256), 0, STREAM, x, idx, w, b, (bf16_t*)y, ld_y, E, eps);
  return DONE;
}

B200_API int b200_glu(void* a, int ld_a, int in_f32, int clear, void* y, int ld_y, int rows, int N, int silu, int f32, void* stream) {
  if (rows <= 0 || N <= 0 || (clear && !in_f32) || (f32 && !in_f32)) return -1;
  for (int r = 0; r < rows; r += 65535) {
    const dim3 grid((N + 255) / 256, rows - r < 65535 ? rows - r : 65535);
    const size_t ao = static_cast<size_t>(r) * ld_a, yo = static_cast<size_t>(r) * ld_y;
#define GO(TI, T, S) launch_k(glu_kernel<TI, T, S>, grid, dim3(256), 0, STREAM, (TI*)a + ao, ld_a, clear, (T*)y + yo, ld_y, N)
    if (f32) { if (silu) GO(float, float, true); else GO(float, float, false); }
    else if (in_f32) { if (silu) GO(float, bf16_t, true); else GO(float, bf16_t, false); }
    else { if (silu) GO(bf16_t, bf16_t, true); else GO(bf16_t, bf16_t, false); }
#undef GO
  }
  return DONE;
}

B200_API int b200_kv_append(const void* in, int ld_in, const float* bias, void* cache, int width, int ld_kv, int cap, const int* pos,
                            const int* row, int T, int in_f32, int f32, void* stream) {
  if (T <= 0 || width <= 0 || (width & 7) || (ld_in & 7) || (ld_kv & 7) || width > ld_kv || cap <= 0 || (f32 && !in_f32)) return -1;
  if ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(bias)) & 15) return -1;
  const long long total = static_cast<long long>(T) * (width / 8);
  if (total > 0x7fffffffll - 256) return -1;
#define GO(TI, T_) launch_k(kv_append_kernel<TI, T_>, dim3(static_cast<unsigned>((total + 255) / 256)), dim3(256), 0, STREAM, (const TI*)in, ld_in, bias, (T_*)cache, width, ld_kv, cap, pos, row, static_cast<int>(total))
  if (f32) GO(float, float);
  else if (in_f32) GO(float, bf16_t);
  else GO(bf16_t, bf16_t);
#undef GO
  return DONE;
}

// n: sequences.  hin / w_gate are only read when the gates are formed here.
B200_API int b200_memory_scan(const void* in, const void* hin, const void* w_gate, void* out, const MemoryArgs* Mp, int n, int in_f32,
                              int f32, void* stream) {
  MemoryArgs M = *Mp;
  if (n <= 0 || n > 65535 || M.H <= 0 || M.dim <= 0 || M.vdim <= 0 || M.ldv < M.vdim || (M.ldv & 3) || !M.state || (f32 && !in_f32)) return -1;
  if (!M.seqs && (!M.pos || !M.row)) return -1;
  if (M.decay ? !M.out32 : (!M.stab || !M.norm_w || !M.gate_bias || !out || (!M.gates && (!hin || !w_gate)))) return -1;
  const int dp = (M.dim + 3) & ~3;
  size_t smem = (3 * dp + 9 * M.ldv + 16) * sizeof(float);
  const size_t st = static_cast<size_t>(M.dim) * M.ldv * sizeof(float);
  M.stage = M.seqs && smem + st <= 220 * 1024;     // otherwise the state stays in global memory
  if (M.stage) smem += st;
  if (smem > 220 * 1024) return -1;
#define GO(TI, T_, G)                                                                                                  \
  {                                                                                                                    \
    if (smem > 48 * 1024 && cudaFuncSetAttribute(memory_scan_kernel<TI, T_, G>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                                 static_cast<int>(smem)) != cudaSuccess) return -3;                     \
    launch_k(memory_scan_kernel<TI, T_, G>, dim3(M.H, n), dim3(256), smem, STREAM, (const TI*)in, (const T_*)hin, (const T_*)w_gate, (T_*)out, M); \
  }
  if (M.decay) {
    if (f32) GO(float, float, false)
    else if (in_f32) GO(float, bf16_t, false)
    else GO(bf16_t, bf16_t, false)
  } else {
    if (f32) GO(float, float, true)
    else if (in_f32) GO(float, bf16_t, true)
    else GO(bf16_t, bf16_t, true)
  }
#undef GO
  return DONE;
}

// mem_f32: the memory outputs are fp32
B200_API int b200_memory_merge(const void* in, const void* mem, void* out, const MergeArgs* Ap, int T, int in_f32, int mem_f32, int f32,
                               void* stream) {
  const MergeArgs A = *Ap;
  if (T <= 0 || A.HR <= 0 || A.rvdim <= 0 || (A.H && (!A.part_o || !A.part_ml || A.splits < 1 || A.splits > 32)) || (f32 && (!in_f32 || !mem_f32))) return -1;
  if (((A.ld_mem | A.ld_in | A.ld_out | A.off_r | A.off_rg) & 7) || ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(mem) | reinterpret_cast<uintptr_t>(out)) & 15)) return -1;
  const int W = A.HR * A.rvdim;
  if (!f32 && !in_f32 && !mem_f32 && A.H == 0 && T >= 256 && (W & 7) == 0 && W <= 16 * 256 && !(reinterpret_cast<uintptr_t>(A.norm_w) & 15)) {
#define GO(G) memory_norm_rows_kernel<G><<<(T + 3) / 4, 128, 0, STREAM>>>((const bf16_t*)in, (const bf16_t*)mem, (bf16_t*)out, A, T)
    if (W <= 4 * 256) GO(4);
    else if (W <= 9 * 256) GO(9);
    else GO(16);
#undef GO
    return DONE;
  }
  const dim3 grid(T, 1 + (A.H + 7) / 8);
#define GO(TI, TM, T_) launch_k(memory_merge_kernel<TI, TM, T_>, grid, dim3(256), 0, STREAM, (const TI*)in, (const TM*)mem, (T_*)out, A)
  if (f32) GO(float, float, float);
  else if (in_f32 && mem_f32) GO(float, float, bf16_t);
  else if (mem_f32) GO(bf16_t, float, bf16_t);
  else GO(bf16_t, bf16_t, bf16_t);
#undef GO
  return DONE;
}
