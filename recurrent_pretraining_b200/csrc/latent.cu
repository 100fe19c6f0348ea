// Kernels of the layered decoder models (latent attention over a per-token latent, fp32 residual stream) other than
// the tensor-core attention tiles:
//   * embed_resid      : token embedding into the fp32 residual stream and its operand-precision copy
//   * latent_prep      : one packed projection row [q | gate | latent]: rotation of the q parts, latent norm, rotation of
//                        the shared key part, append to the ring cache and to the step's key stream
//   * latent_absorb    : the decode form of the same step; q is also carried through the key up-projection, so that the
//                        scores are taken against the cached latents directly
//   * window_attention : softmax over the keys of a sliding window, one query row per (token, head); generic in every
//                        size, 32-bit throughout (step streams and ring caches)
//   * latent_expand    : merge of the decode attention's key splits, value up-projection, output gate
//   * rms_residual     : x += mult * rmsnorm(a + bias) * w on the fp32 residual stream
//   * bias_act, rmsnorm_rows, gather_rows, sgemm_nt (true fp32 matrix product)
// Storage types: bf16 (serving) or fp32; arithmetic is fp32.  This file is built without fast-math approximations.
#include "rowops.cuh"

namespace b200 {

// ------------------------------------------------------------------------------------------------ embedding
template <typename T>
__global__ void __launch_bounds__(128)
embed_resid_kernel(const long long* __restrict__ tok, const T* __restrict__ table, float* __restrict__ x,
                   T* __restrict__ xb, int E, int ld_table, int ld_xb, float scale, long long vocab, int* err) {
  const size_t t = blockIdx.x;
  long long id = tok[t];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0) atomicCAS(err, 0, ERR_BAD_INDEX);
  const T* src = table + static_cast<size_t>(ok ? id : 0) * ld_table;
  for (int i = threadIdx.x; i < E; i += 128) {
    const float v = ok ? ldf(src + i) * scale : 0.f;
    x[t * E + i] = v;
    if (xb) stf(xb + t * ld_xb + i, v);
  }
}

// ------------------------------------------------------------------------------------------------ latent rows
struct LatentRow {
  // projection row: q at column 0 (head by head [dim | rot]), gate at off_g, latent [rank | rot] at off_d
  int ld_in, off_g, off_d;
  int H, dim, rot, rank, vdim;
  int rank_pad, ld_lat;           // latent row: [c (rank) | 0 .. rank_pad | rotated key part (rot) | 0 .. ld_lat]
  int cap;                        // ring slots of one sequence row
  int own;                        // this layer has a latent projection of its own
  float eps;
  const float* norm_w;            // [rank]
  const float* cosT;              // [positions, rot / 2], scaled
  const float* sinT;
  const int* pos;                 // [T]
  const int* row;                 // [T] cache row
};

// latent part of one token -> cache row `dst_cache` (or null) and stream row `dst_stream` (or null)
template <typename TI, typename T, int THREADS>
__device__ __forceinline__ void latent_append(const LatentRow& L, const TI* in, int p, T* dst_cache, T* dst_stream, float* red) {
  const TI* d = in + L.off_d;
  float ss = 0.f;
  for (int i = threadIdx.x; i < L.rank; i += THREADS) {
    const float v = ldf(d + i);
    ss += v * v;
  }
  const float rstd = 1.f / sqrtf(block_total<THREADS>(ss, red) / static_cast<float>(L.rank) + L.eps);
  for (int i = threadIdx.x; i < L.ld_lat; i += THREADS) {
    float v = 0.f;
    if (i < L.rank) {
      v = ldf(d + i) * rstd * L.norm_w[i];
    } else if (i >= L.rank_pad && i < L.rank_pad + L.rot) {
      const int j = i - L.rank_pad, pr = j >> 1;
      const float u = ldf(d + L.rank + (j & ~1)), w = ldf(d + L.rank + (j | 1));
      const float c = L.cosT[static_cast<size_t>(p) * (L.rot >> 1) + pr], s = L.sinT[static_cast<size_t>(p) * (L.rot >> 1) + pr];
      v = (j & 1) ? w * c + u * s : u * c - w * s;
    }
    if (dst_cache) stf(dst_cache + i, v);
    if (dst_stream) stf(dst_stream + i, v);
  }
}

// One CTA per token of a packed step.  Rotates the q parts in place; appends the latent row to the stream at sidx[t] and,
// for the last `cap` tokens of the sequence's portion (end[t] = position after its last token), to the ring (if there is one).
template <typename T>
__global__ void __launch_bounds__(128)
latent_prep_kernel(T* __restrict__ in, LatentRow L, const int* __restrict__ sidx, const int* __restrict__ end,
                   T* __restrict__ cache, T* __restrict__ stream) {
  __shared__ float red[4];
  const size_t t = blockIdx.x;
  T* r = in + t * L.ld_in;
  const int p = L.pos[t], half = L.rot >> 1, hd = L.dim + L.rot;
  const float* ct = L.cosT + static_cast<size_t>(p) * half;
  const float* st = L.sinT + static_cast<size_t>(p) * half;
  if ((L.dim & 1) == 0) {                           // pairs are aligned to two elements
#pragma unroll 4
    for (int i = threadIdx.x; i < L.H * half; i += 128) {
      const int h = i / half, j = i - h * half;
      T* q = r + h * hd + L.dim + 2 * j;
      const float2 f = ld2(q);
      const float c = ct[j], s = st[j];
      st2(q, make_float2(f.x * c - f.y * s, f.y * c + f.x * s));
    }
  } else {
    for (int i = threadIdx.x; i < L.H * half; i += 128) {
      const int h = i / half, j = i - h * half;
      T* q = r + h * hd + L.dim + 2 * j;
      const float u = ldf(q), v = ldf(q + 1), c = ct[j], s = st[j];
      stf(q, u * c - v * s);
      stf(q + 1, v * c + u * s);
    }
  }
  if (L.own) {
    T* dst = cache && p >= end[t] - L.cap ? cache + (static_cast<size_t>(L.row[t]) * L.cap + p % L.cap) * L.ld_lat : nullptr;
    latent_append<T, T, 128>(L, r, p, dst, stream + static_cast<size_t>(sidx[t]) * L.ld_lat, red);
  }
}

// Four neighbouring weights as they lie in memory.
template <typename T> struct Raw4;
template <> struct Raw4<float> {
  float4 q;
  __device__ __forceinline__ void load(const float* p) { q = *reinterpret_cast<const float4*>(p); }
  __device__ __forceinline__ void get(float (&v)[4]) const { v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
};
template <> struct Raw4<__nv_bfloat16> {
  uint2 q;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { q = *reinterpret_cast<const uint2*>(p); }
  __device__ __forceinline__ void get(float (&v)[4]) const {
    const float2 a = unpack_bf16x2(q.x), b = unpack_bf16x2(q.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
};

// Decode: in [B, ld_in] (fp32 accumulator or operand precision, not modified).  Three kinds of CTAs:
//   [0, n_lat)               row b's latent append (layers with latents of their own)
//   [n_lat, n_lat + n_rot)   rotated and padding columns of qlat [B, H, ld_lat], one pair of columns per thread
//   the others               (head, 128 latent columns, 8 rows) tiles of qlat[b, h, r] = sum_d W_uk[h * dim + d, r] q[b, h, d]
constexpr int ABS_ROWS = 8, ABS_COLS = 128;
template <typename TI, typename T>
__global__ void __launch_bounds__(256, 3)
latent_absorb_kernel(const TI* __restrict__ in, LatentRow L, const T* __restrict__ w_uk, int ldw, T* __restrict__ cache,
                     T* __restrict__ qlat, int B, int n_lat, int n_rot) {
  pdl_trigger();
  extern __shared__ float sm[];
  const int hd = L.dim + L.rot, half = L.rot >> 1;
  int id = blockIdx.x;
  if (id < n_lat) {
    pdl_wait();
    const int b = id, p = L.pos[b];
    latent_append<TI, T, 256>(L, in + static_cast<size_t>(b) * L.ld_in, p,
                              cache + (static_cast<size_t>(L.row[b]) * L.cap + p % L.cap) * L.ld_lat, static_cast<T*>(nullptr), sm);
    return;
  }
  id -= n_lat;
  if (id < n_rot) {
    pdl_wait();
    const int pairs = (L.ld_lat - L.rank_pad) >> 1;
    const int i = id * 256 + threadIdx.x;
    if (i >= B * L.H * pairs) return;
    const int j = i % pairs, bh = i / pairs, b = bh / L.H, h = bh - b * L.H;
    T* dst = qlat + static_cast<size_t>(bh) * L.ld_lat;
    float v0 = 0.f, v1 = 0.f;
    if (j < half) {
      const TI* q = in + static_cast<size_t>(b) * L.ld_in + h * hd + L.dim + 2 * j;
      const size_t t = static_cast<size_t>(L.pos[b]) * half + j;
      const float u = ldf(q), w = ldf(q + 1), c = L.cosT[t], s = L.sinT[t];
      v0 = u * c - w * s;
      v1 = w * c + u * s;
    }
    stf(dst + L.rank_pad + 2 * j, v0);
    stf(dst + L.rank_pad + 2 * j + 1, v1);
    for (int c = L.rank + j; c < L.rank_pad; c += pairs) stf(dst + c, 0.f);
    return;
  }
  id -= n_rot;
  const int cols = (L.rank + ABS_COLS - 1) / ABS_COLS;
  const int rc = id % cols;
  id /= cols;
  const int h = id % L.H, b0 = (id / L.H) * ABS_ROWS;
  const int nb = min(ABS_ROWS, B - b0);
  float* qs = sm;                                  // [dim][ABS_ROWS]
  float* part = sm + ABS_ROWS * ((L.dim + 3) & ~3);   // [8][ABS_ROWS][ABS_COLS]
  const int tx = threadIdx.x & 31, grp = threadIdx.x >> 5;   // four columns per thread, eight groups over d
  const int r = rc * ABS_COLS + 4 * tx;
  const bool live = r < L.rank;                    // weight rows are padded to eight: columns up to r + 3 exist
  const T* wp = w_uk + static_cast<size_t>(h) * L.dim * ldw + (live ? r : 0);
  constexpr int U = 16;                            // weight rows in flight per thread; the first ones do not wait for q
  Raw4<T> w[U];
#pragma unroll
  for (int u = 0; u < U; ++u)
    if (grp + 8 * u < L.dim) w[u].load(wp + static_cast<size_t>(grp + 8 * u) * ldw);
  pdl_wait();
  for (int b = grp; b < ABS_ROWS; b += 8)          // warp b reads row b
    for (int d = tx; d < L.dim; d += 32)
      qs[d * ABS_ROWS + b] = b < nb ? ldf(in + static_cast<size_t>(b0 + b) * L.ld_in + h * hd + d) : 0.f;
  __syncthreads();
  float acc[ABS_ROWS][4];
#pragma unroll
  for (int b = 0; b < ABS_ROWS; ++b)
#pragma unroll
    for (int k = 0; k < 4; ++k) acc[b][k] = 0.f;
#pragma unroll 1
  for (int d0 = grp; d0 < L.dim; d0 += 8 * U) {
    if (d0 != grp) {
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (d0 + 8 * u < L.dim) w[u].load(wp + static_cast<size_t>(d0 + 8 * u) * ldw);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (d0 + 8 * u < L.dim) {
        float q[8], wf[4];
        ld8(qs + (d0 + 8 * u) * ABS_ROWS, q);
        w[u].get(wf);
#pragma unroll
        for (int b = 0; b < ABS_ROWS; ++b)
#pragma unroll
          for (int k = 0; k < 4; ++k) acc[b][k] += q[b] * wf[k];
      }
    }
  }
#pragma unroll
  for (int b = 0; b < ABS_ROWS; ++b)
    *reinterpret_cast<float4*>(&part[(grp * ABS_ROWS + b) * ABS_COLS + 4 * tx]) = make_float4(acc[b][0], acc[b][1], acc[b][2], acc[b][3]);
  __syncthreads();
  for (int i = threadIdx.x; i < nb * ABS_COLS; i += 256) {
    const int b = i / ABS_COLS, c = i - b * ABS_COLS;
    if (rc * ABS_COLS + c >= L.rank) continue;
    float v = 0.f;
#pragma unroll
    for (int g = 0; g < 8; ++g) v += part[(g * ABS_ROWS + b) * ABS_COLS + c];
    stf(qlat + (static_cast<size_t>(b0 + b) * L.H + h) * L.ld_lat + rc * ABS_COLS + c, v);
  }
}

// dst[dst_idx[i], :] = src[src_idx[i], :], rows of `bytes` (a multiple of 16) bytes
__global__ void __launch_bounds__(128)
gather_rows_kernel(const uint4* __restrict__ src, const int* __restrict__ src_idx, uint4* __restrict__ dst,
                   const int* __restrict__ dst_idx, int vec) {
  const uint4* s = src + static_cast<size_t>(src_idx[blockIdx.x]) * vec;
  uint4* d = dst + static_cast<size_t>(dst_idx[blockIdx.x]) * vec;
  for (int i = threadIdx.x; i < vec; i += 128) d[i] = s[i];
}

// ------------------------------------------------------------------------------------------------ attention (generic)
struct WindowAttn {
  // score(t, h, key) = q[t, h, :d1] . k1[key, h, :] + q[t, h, d1:] . k2[key, :]
  int H, d1, d2, vdim, window, splits;
  float scale;
  int q_stride, q_head;           // elements
  int k1_stride, k1_head, k2_stride, v_stride, v_head;
  const int* sidx;                // stream form: key index of the query itself ...
  const int* kbase;               // ... and of the first key of its sequence
  const int* pos;                 // ring form: position of the query ...
  const int* row;                 // ... and its cache row (key of position p: row * cap + p % cap)
  int cap;
  // stream form: normalised, gated output; ring form (splits > 0 partials): unnormalised fp32 partials
  int gate_ld, out_ld;
  float* part_o;                  // [T, H, splits, vdim padded to eight]
  float* part_ml;                 // [T, H, splits, 2] (max in natural-log units, sum)
  int group;                      // query heads per key / value head
  // distance bias (null: none): score += bias[h * bias_len + min(distance, bias_len - 1)]
  const float* bias;
  int bias_len;
  // query temperature (0: none): scores are multiplied by 1 + coef * ln(floor((position + 1) / every) + 1)
  int temp_every;
  float temp_coef;
  int head_gate;                  // stream form: one gate per head (gate row [H]) instead of one per output; no gate array: none
  float gate_mult;                // factor on the gated output
  float softcap;                  // 0: none; otherwise score = softcap * tanh(score / softcap)
  int chunk;                      // ring form, not 0: the query sees its chunk of that many positions instead of a window
  const float* sink;              // [H] stream form, null: none; exp(sink) is one more term of the softmax's denominator
  int keep;                       // the first `keep` keys of a sequence are visible beside the window (not with chunks)
};

// CTA of four warps per (token, head, key split); a warp takes 32 keys at a time: one key per lane for the scores, one
// value column per lane for the weighted sum.
template <typename T>
__global__ void __launch_bounds__(128)
window_attn_kernel(const T* __restrict__ q, const T* __restrict__ k1, const T* __restrict__ k2, const T* __restrict__ v,
                   const T* __restrict__ gate, T* __restrict__ out, const WindowAttn A) {
  extern __shared__ float sm[];
  const int dk = A.d1 + A.d2;
  float* qs = sm;                                   // [dk]
  float* ps = sm + dk;                              // [4][32]
  float* os = ps + 128;                             // [4][vdim]
  float* ml = os + 4 * A.vdim;                      // [4][2]
  const int t = blockIdx.x, h = blockIdx.y, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* qp = q + static_cast<size_t>(t) * A.q_stride + static_cast<size_t>(h) * A.q_head;
  for (int i = threadIdx.x; i < dk; i += 128) qs[i] = ldf(qp + i);
  for (int i = threadIdx.x; i < 4 * A.vdim; i += 128) os[i] = 0.f;
  __syncthreads();
  const bool ring = A.pos != nullptr;
  const int last = ring ? A.pos[t] : A.sidx[t];
  const int first = ring && A.chunk ? last - last % A.chunk : max(ring ? 0 : A.kbase[t], last - A.window + 1);
  // visible keys are counted: kept ones in front of the window, then the window
  const int origin = ring ? 0 : A.kbase[t], kept = A.chunk ? 0 : min(A.keep, first - origin), nkeys = kept + last - first + 1;
  const size_t ring0 = ring ? static_cast<size_t>(A.row[t]) * A.cap : 0;
  const int nchunk = (nkeys - 1) / 32 + 1;
  auto key_of = [&](int e) -> size_t {
    const int j = e < kept ? origin + e : first + (e - kept);
    return ring ? ring0 + ring_slot(j, A.cap, A.keep) : static_cast<size_t>(j);
  };
  const int hk = h / A.group;
  float scale = A.scale;
  if (A.temp_every > 0) scale *= query_temperature(ring ? last : last - A.kbase[t], A.temp_every, A.temp_coef);
  const float* bias = A.bias ? A.bias + static_cast<size_t>(h) * A.bias_len : nullptr;
  float m = -INFINITY, l = 0.f;
  float* op = os + warp * A.vdim;
  float* pp = ps + warp * 32;
  for (int c = split * 4 + warp; c < nchunk; c += 4 * A.splits) {
    const int j0 = c * 32, n = min(32, nkeys - j0);
    float s = -INFINITY;
    if (lane < n) {
      const size_t key = key_of(j0 + lane);
      const T* a = k1 + key * A.k1_stride + static_cast<size_t>(hk) * A.k1_head;
      s = 0.f;
      for (int i = 0; i < A.d1; ++i) s += qs[i] * ldf(a + i);
      if (A.d2) {
        const T* b = k2 + key * A.k2_stride;
        for (int i = 0; i < A.d2; ++i) s += qs[A.d1 + i] * ldf(b + i);
      }
      s *= scale;
      if (bias) s += bias[min(last - first - (j0 + lane), A.bias_len - 1)];     // not with kept keys
      if (A.softcap > 0.f) s = A.softcap * tanhf(s / A.softcap);
    }
    const float mn = fmaxf(m, warp_max(s));
    const float p = expf(s - mn), alpha = expf(m - mn);
    l = l * alpha + warp_sum(p);
    m = mn;
    pp[lane] = p;
    __syncwarp();
    for (int d = lane; d < A.vdim; d += 32) {
      float o = op[d] * alpha;
      for (int k = 0; k < n; ++k) {
        const size_t key = key_of(j0 + k);
        o += pp[k] * ldf(v + key * A.v_stride + static_cast<size_t>(hk) * A.v_head + d);
      }
      op[d] = o;
    }
    __syncwarp();
  }
  if (lane == 0) { ml[2 * warp] = m; ml[2 * warp + 1] = l; }
  __syncthreads();
  float mm = -INFINITY, ll = 0.f, wgt[4];
#pragma unroll
  for (int w = 0; w < 4; ++w) mm = fmaxf(mm, ml[2 * w]);
  const float sink = A.sink ? A.sink[h] : -INFINITY;
  if (A.sink) {                                     // stream form: some key is visible
    mm = fmaxf(mm, sink);
    ll = expf(sink - mm);
  }
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    wgt[w] = ml[2 * w] == -INFINITY ? 0.f : expf(ml[2 * w] - mm);
    ll += wgt[w] * ml[2 * w + 1];
  }
  const float inv = 1.f / ll;
  for (int d = threadIdx.x; d < A.vdim; d += 128) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) o += wgt[w] * os[w * A.vdim + d];
    if (A.part_o) {
      const size_t pi = (static_cast<size_t>(t) * A.H + h) * A.splits + split;
      A.part_o[pi * ((A.vdim + 7) & ~7) + d] = o;
      if (d == 0) { A.part_ml[2 * pi] = mm; A.part_ml[2 * pi + 1] = ll; }
    } else {
      const float g = gate ? sigmoid_f(ldf(gate + static_cast<size_t>(t) * A.gate_ld + (A.head_gate ? h : h * A.vdim + d))) : 1.f;
      stf(out + static_cast<size_t>(t) * A.out_ld + h * A.vdim + d, o * inv * (g * A.gate_mult));
    }
  }
}

// Sum over the lanes of a warp of N values per lane (N a power of two <= 32) by halving exchanges: afterwards lane l holds the
// total of value l % N.
template <int N>
__device__ __forceinline__ float warp_sum_many(float (&v)[N]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int off = 16; off >= N; off >>= 1) {
#pragma unroll
    for (int k = 0; k < N; ++k) v[k] += __shfl_xor_sync(0xffffffffu, v[k], off);
  }
#pragma unroll
  for (int off = N / 2; off > 0; off >>= 1) {
#pragma unroll
    for (int k = 0; k < off; ++k) {
      const bool up = lane & off;
      const float send = up ? v[k] : v[k + off], keep = up ? v[k + off] : v[k];
      v[k] = keep + __shfl_xor_sync(0xffffffffu, send, off);
    }
  }
  return v[0];
}

// out[b, h * vdim + v] = sigmoid(gate) * sum_r W_uv[h * vdim + v, r] o[b, h, r], o = merged key splits (partial rows are
// padded to eight columns).
// CTA: (head, 32 values, ROWS rows); a warp forms four values of all its rows at once.
constexpr int EXP_COLS = 32;
template <typename TI, typename T, int ROWS>
__global__ void __launch_bounds__(256, sizeof(T) == 2 ? 3 : 2)
latent_expand_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int splits,
                     const T* __restrict__ w_uv, int ldw, const TI* __restrict__ gate, int gate_ld, T* __restrict__ out,
                     int out_ld, int B, int H, int rank, int vdim) {
  pdl_trigger();
  extern __shared__ float os[];                    // [ROWS][rank padded to eight]
  const int h = blockIdx.x, v0 = blockIdx.y * EXP_COLS, b0 = blockIdx.z * ROWS;
  const int nb = min(ROWS, B - b0), rs = (rank + 7) & ~7;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // four weight rows per warp; the pieces of the first columns do not wait for the attention
  const int vw = v0 + warp * 4;
  const T* wr = w_uv + (static_cast<size_t>(h) * vdim + vw) * ldw;
  constexpr int PRE = 2;                           // 4-column pieces per row held ahead: 32 lanes x 4 x PRE columns
  Raw4<T> w[4][PRE];
  auto load_w = [&](int r0) {
#pragma unroll
    for (int k = 0; k < 4; ++k)
#pragma unroll
      for (int e = 0; e < PRE; ++e) {
        const int r = r0 + 128 * e + 4 * lane;
        if (vw + k < vdim && r < rs) w[k][e].load(wr + static_cast<size_t>(k) * ldw + r);
      }
  };
  load_w(0);
  pdl_wait();
  float gv = 0.f;                                  // gate of the one result this lane stores in the end
  {
    const int b = lane >> 2, v = vw + (lane & 3);
    if (lane < 4 * ROWS && b < nb && v < vdim) gv = ldf(gate + static_cast<size_t>(b0 + b) * gate_ld + h * vdim + v);
  }
  {                                                // merge: warps b * WPR .. of row b; lane s holds the weight of split s
    constexpr int WPR = 8 / ROWS;
    const int b = warp / WPR;
    const size_t base = (static_cast<size_t>(b0 + (b < nb ? b : 0)) * H + h) * splits;
    const float2 e = lane < splits ? *reinterpret_cast<const float2*>(part_ml + (base + lane) * 2) : make_float2(-INFINITY, 0.f);
    const float mm = warp_max(e.x);
    const float a = e.x == -INFINITY ? 0.f : expf(e.x - mm);
    const float mine = b < nb ? a / warp_sum(a * e.y) : 0.f;
    const float* p = part_o + base * rs;
    for (int r0 = 128 * (warp % WPR); r0 < rs; r0 += 128 * WPR) {   // uniform over the warp
      const int r = r0 + 4 * lane;
      float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
      for (int s = 0; s < splits; ++s) {
        const float w = __shfl_sync(0xffffffffu, mine, s);
        float x[4] = {0.f, 0.f, 0.f, 0.f};
        if (r < rs) ld4(p + static_cast<size_t>(s) * rs + r, x);
#pragma unroll
        for (int k = 0; k < 4; ++k) o[k] += w != 0.f ? w * x[k] : 0.f;   // an empty split's partial is not initialised
      }
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (r + k >= rank) o[k] = 0.f;             // neither are the padding columns
      if (r < rs) *reinterpret_cast<float4*>(os + b * rs + r) = make_float4(o[0], o[1], o[2], o[3]);
    }
  }
  __syncthreads();
  float acc[4 * ROWS];
#pragma unroll
  for (int i = 0; i < 4 * ROWS; ++i) acc[i] = 0.f;
#pragma unroll 1
  for (int r0 = 0; r0 < rs; r0 += 128 * PRE) {     // weight rows are padded to eight with zeros
    if (r0) load_w(r0);
#pragma unroll
    for (int e = 0; e < PRE; ++e) {
      const int r = r0 + 128 * e + 4 * lane;
      if (r >= rs) continue;
      float wf[4][4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        w[k][e].get(wf[k]);
        if (vw + k >= vdim) wf[k][0] = wf[k][1] = wf[k][2] = wf[k][3] = 0.f;
      }
#pragma unroll
      for (int b = 0; b < ROWS; ++b) {
        float o[4];
        ld4(os + b * rs + r, o);
#pragma unroll
        for (int k = 0; k < 4; ++k)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[b * 4 + k] += wf[k][j] * o[j];
      }
    }
  }
  const float s = warp_sum_many<4 * ROWS>(acc);
  const int b = lane >> 2, v = vw + (lane & 3);
  if (lane < 4 * ROWS && b < nb && v < vdim) {
    stf(out + static_cast<size_t>(b0 + b) * out_ld + h * vdim + v, s * sigmoid_f(gv));
  }
}

// ------------------------------------------------------------------------------------------------ residual
// x += mult * (s / rms(s)) * w with s = a + bias; xb = x in operand precision.  One CTA per row.  `clear`: a is the
// accumulator of a stream-K GEMM and is handed back zeroed; zero[row, :nzero] is a second accumulator (consumed by earlier
// kernels) that is re-armed here.
template <typename TI, typename T, int NV>
__global__ void __launch_bounds__(256)
rms_residual_vec_kernel(TI* __restrict__ a, int ld_a, int clear, const float* __restrict__ bias, const float* __restrict__ w,
                        float* __restrict__ x, T* __restrict__ xb, int ld_xb, int E, float eps, float mult,
                        float* __restrict__ zero, int nzero) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const size_t row = blockIdx.x;
  const int nvec = E >> 3;
  TI* ar = a + row * ld_a;
  float s[NV][8], xv[NV][8];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i < nvec) {
      ld8(ar + 8 * i, s[k]);
      ld8(x + row * E + 8 * i, xv[k]);
      if (bias) {
        float b[8];
        ld8(bias + 8 * i, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) s[k][j] += b[j];
      }
      if (clear) clear8(ar + 8 * i);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += s[k][j] * s[k][j];
    }
  }
  for (int i = threadIdx.x; i < nzero; i += 256) zero[row * nzero + i] = 0.f;
  const float r = mult / sqrtf(block_total<256>(ss, red) / static_cast<float>(E) + eps);
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i < nvec) {
      float wv[8];
      ld8(w + 8 * i, wv);
#pragma unroll
      for (int j = 0; j < 8; ++j) xv[k][j] += s[k][j] * r * wv[j];
      st8(x + row * E + 8 * i, xv[k]);
      st8(xb + row * ld_xb + 8 * i, xv[k]);
    }
  }
}

template <typename TI, typename T>
__global__ void __launch_bounds__(256)
rms_residual_kernel(TI* __restrict__ a, int ld_a, int clear, const float* __restrict__ bias, const float* __restrict__ w,
                    float* __restrict__ x, T* __restrict__ xb, int ld_xb, int E, float eps, float mult,
                    float* __restrict__ zero, int nzero) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const size_t row = blockIdx.x;
  TI* ar = a + row * ld_a;
  float ss = 0.f;
  for (int i = threadIdx.x; i < E; i += 256) {
    const float s = ldf(ar + i) + (bias ? bias[i] : 0.f);
    ss += s * s;
  }
  for (int i = threadIdx.x; i < nzero; i += 256) zero[row * nzero + i] = 0.f;
  const float r = mult / sqrtf(block_total<256>(ss, red) / static_cast<float>(E) + eps);
  for (int i = threadIdx.x; i < E; i += 256) {
    const float s = ldf(ar + i) + (bias ? bias[i] : 0.f);
    if (clear) stf(ar + i, 0.f);
    const float v = x[row * E + i] + s * r * w[i];
    x[row * E + i] = v;
    stf(xb + row * ld_xb + i, v);
  }
}

// y[i] = mult * rmsnorm(x[idx[i]]) * (w + w_add) in operand precision
template <typename T>
__global__ void __launch_bounds__(256)
rmsnorm_rows_kernel(const float* __restrict__ x, const int* __restrict__ idx, const float* __restrict__ w, T* __restrict__ y,
                    int ld_y, int E, float eps, float w_add, float mult) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const float* xr = x + static_cast<size_t>(idx ? idx[blockIdx.x] : static_cast<int>(blockIdx.x)) * E;
  float ss = 0.f;
  for (int i = threadIdx.x; i < E; i += 256) ss += xr[i] * xr[i];
  const float r = 1.f / sqrtf(block_total<256>(ss, red) / static_cast<float>(E) + eps);
  for (int i = threadIdx.x; i < E; i += 256) stf(y + static_cast<size_t>(blockIdx.x) * ld_y + i, xr[i] * r * (w[i] + w_add) * mult);
}

// y = act(a + bias); act 0: none, 1: relu^2.  `clear` as above.
template <typename TI, typename T>
__global__ void __launch_bounds__(256)
bias_act_kernel(TI* __restrict__ a, int ld_a, int clear, const float* __restrict__ bias, T* __restrict__ y, int ld_y, int N, int act) {
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.y;
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i >= N) return;
  float v = ldf(a + row * ld_a + i) + (bias ? bias[i] : 0.f);
  if (clear) stf(a + row * ld_a + i, 0.f);
  if (act == 1) {
    v = fmaxf(v, 0.f);
    v *= v;
  }
  stf(y + row * ld_y + i, v);
}

// ------------------------------------------------------------------------------------------------ fp32 matrix product
// C[M, N] = act(A[M, K] B[N, K]^T + bias) in fp32 (FMA pipe): 64 x 64 tile per 256 threads, 4 x 4 per thread.  Grouped: tile i of the
// first *n_tiles row tiles is multiplied with rows [group[i] N, (group[i] + 1) N) of B.
constexpr int SG = 64, SGK = 16;
__global__ void __launch_bounds__(256)
sgemm_nt_kernel(const float* __restrict__ A, const float* __restrict__ B, const float* __restrict__ bias, float* __restrict__ C,
                int M, int N, int K, int lda, int ldb, int ldc, int act, int act_lo, int act_hi, const int* __restrict__ group,
                const int* __restrict__ n_tiles) {
  if (group) {
    if (static_cast<int>(blockIdx.x) >= *n_tiles) return;
    B += static_cast<size_t>(group[blockIdx.x]) * N * ldb;
  }
  __shared__ float as[SGK][SG + 4], bs[SGK][SG + 4];
  const int m0 = blockIdx.x * SG, n0 = blockIdx.y * SG;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += SGK) {
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int i = threadIdx.x + u * 256, r = i >> 4, c = i & 15;
      as[c][r] = (m0 + r < M && k0 + c < K) ? A[static_cast<size_t>(m0 + r) * lda + k0 + c] : 0.f;
      bs[c][r] = (n0 + r < N && k0 + c < K) ? B[static_cast<size_t>(n0 + r) * ldb + k0 + c] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SGK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&as[k][4 * ty]), b = *reinterpret_cast<const float4*>(&bs[k][4 * tx]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += av[i] * bv[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + 4 * ty + i;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + 4 * tx + j;
      if (m >= M || n >= N) continue;
      float v = acc[i][j] + (bias ? bias[n] : 0.f);
      if (act == 1) {
        v = fmaxf(v, 0.f);
        v *= v;
      } else if (act == 2 && n >= act_lo && n < act_hi) {
        v = silu_f(v);
      }
      C[static_cast<size_t>(m) * ldc + n] = v;
    }
  }
}

}  // namespace b200

using namespace b200;
typedef __nv_bfloat16 bf16_t;
#define STREAM reinterpret_cast<cudaStream_t>(stream)
#define DONE (cudaGetLastError() == cudaSuccess ? 0 : -2)

// Every `f32` argument: the operand storage type is fp32 instead of bf16; `in_f32`: the GEMM output is fp32.

B200_API int b200_embed_resid(const long long* tok, const void* table, float* x, void* xb, int T, int E, int ld_table, int ld_xb,
                              float scale, long long vocab, int f32, int* err, void* stream) {
  if (T <= 0 || E <= 0 || vocab <= 0 || ld_table < E || (xb && ld_xb < E)) return -1;
  if (f32) embed_resid_kernel<float><<<T, 128, 0, STREAM>>>(tok, (const float*)table, x, (float*)xb, E, ld_table, ld_xb, scale, vocab, err);
  else embed_resid_kernel<bf16_t><<<T, 128, 0, STREAM>>>(tok, (const bf16_t*)table, x, (bf16_t*)xb, E, ld_table, ld_xb, scale, vocab, err);
  return DONE;
}

static bool latent_row_ok(const LatentRow& L) {
  return L.H > 0 && L.dim > 0 && L.rot > 0 && !(L.rot & 1) && L.rank > 0 && L.rank_pad >= L.rank && !(L.rank_pad & 1) &&
         L.ld_lat >= L.rank_pad + L.rot && !(L.ld_lat & 1) && L.cap > 0;
}

B200_API int b200_latent_prep(void* in, const LatentRow* Lp, const int* sidx, const int* end, void* cache, void* stream_buf, int T,
                              int f32, void* stream) {
  const LatentRow L = *Lp;
  if (T <= 0 || !latent_row_ok(L) || (L.own && (!stream_buf || !sidx || !end))) return -1;
  if (f32) latent_prep_kernel<float><<<T, 128, 0, STREAM>>>((float*)in, L, sidx, end, (float*)cache, (float*)stream_buf);
  else latent_prep_kernel<bf16_t><<<T, 128, 0, STREAM>>>((bf16_t*)in, L, sidx, end, (bf16_t*)cache, (bf16_t*)stream_buf);
  return DONE;
}

B200_API int b200_latent_absorb(const void* in, const LatentRow* Lp, const void* w_uk, int ldw, void* cache, void* qlat, int B,
                                int in_f32, int f32, void* stream) {
  const LatentRow L = *Lp;
  if (B <= 0 || !latent_row_ok(L) || (ldw & 7) || ldw < L.rank || (reinterpret_cast<uintptr_t>(w_uk) & 15) || (L.own && !cache) || (f32 && !in_f32)) return -1;
  const int cols = (L.rank + ABS_COLS - 1) / ABS_COLS;
  const int n_lat = L.own ? B : 0, n_rot = (B * L.H * ((L.ld_lat - L.rank_pad) / 2) + 255) / 256;
  const dim3 grid(n_lat + n_rot + cols * L.H * ((B + ABS_ROWS - 1) / ABS_ROWS));
  const size_t smem = (ABS_ROWS * ((L.dim + 3) & ~3) + 8 * ABS_ROWS * ABS_COLS) * sizeof(float);
  if (smem > 200 * 1024) return -1;
#define GO(TI, T)                                                                                                      \
  {                                                                                                                    \
    if (smem > 48 * 1024 && cudaFuncSetAttribute(latent_absorb_kernel<TI, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                                 static_cast<int>(smem)) != cudaSuccess) return -3;                     \
    launch_k(latent_absorb_kernel<TI, T>, grid, dim3(256), smem, STREAM, (const TI*)in, L, (const T*)w_uk, ldw, (T*)cache, (T*)qlat, B, n_lat, n_rot); \
  }
  if (f32) GO(float, float)
  else if (in_f32) GO(float, bf16_t)
  else GO(bf16_t, bf16_t)
#undef GO
  return DONE;
}

B200_API int b200_gather_rows(const void* src, const int* src_idx, void* dst, const int* dst_idx, int n, int row_bytes, void* stream) {
  if (n <= 0) return 0;
  if (row_bytes & 15) return -1;
  gather_rows_kernel<<<n, 128, 0, STREAM>>>((const uint4*)src, src_idx, (uint4*)dst, dst_idx, row_bytes / 16);
  return DONE;
}

B200_API int b200_window_attention(const void* q, const void* k1, const void* k2, const void* v, const void* gate, void* out,
                                   const WindowAttn* Ap, int T, int f32, void* stream) {
  const WindowAttn A = *Ap;
  if (T <= 0 || A.H <= 0 || A.H > 65535 || A.group <= 0 || A.H % A.group || (A.bias && A.bias_len <= 0) || A.d1 <= 0 || A.d2 < 0 || A.vdim <= 0 || A.window <= 0 || A.splits < 1 || A.splits > 32) return -1;
  if (A.pos ? (!A.row || A.cap <= 0 || A.cap < A.window || !A.part_o || !A.part_ml || A.sink) : (!A.sidx || !A.kbase || A.splits != 1 || A.part_o || A.chunk || !out))
    return -1;
  if (A.softcap < 0.f || A.chunk < 0 || A.keep < 0 || (A.keep && (A.bias || A.chunk || A.temp_every > 0))) return -1;
  const size_t smem = (A.d1 + A.d2 + 128 + 4 * A.vdim + 8) * sizeof(float);
  if (smem > 200 * 1024) return -1;
  const dim3 grid(T, A.H, A.splits);
#define GO(T_)                                                                                                         \
  {                                                                                                                    \
    if (smem > 48 * 1024 && cudaFuncSetAttribute(window_attn_kernel<T_>, cudaFuncAttributeMaxDynamicSharedMemorySize,    \
                                                 static_cast<int>(smem)) != cudaSuccess) return -3;                     \
    window_attn_kernel<T_><<<grid, 128, smem, STREAM>>>((const T_*)q, (const T_*)k1, (const T_*)k2, (const T_*)v,        \
                                                        (const T_*)gate, (T_*)out, A);                                  \
  }
  if (f32) GO(float) else GO(bf16_t)
#undef GO
  return DONE;
}

B200_API int b200_latent_expand(const float* part_o, const float* part_ml, int splits, const void* w_uv, int ldw, const void* gate,
                                int gate_ld, void* out, int out_ld, int B, int H, int rank, int vdim, int in_f32, int f32, void* stream) {
  if (B <= 0 || splits < 1 || splits > 32 || (ldw & 7) || ldw < rank || (reinterpret_cast<uintptr_t>(w_uv) & 15) || (f32 && !in_f32)) return -1;
  const int rows = B >= 8 ? 8 : (B > 1 ? 4 : 1);
  const dim3 grid(H, (vdim + EXP_COLS - 1) / EXP_COLS, (B + rows - 1) / rows);
  const size_t smem = rows * ((rank + 7) & ~7) * sizeof(float);
  if (smem > 200 * 1024) return -1;
#define GO2(TI, T, R)                                                                                                  \
  {                                                                                                                    \
    if (smem > 40 * 1024 && cudaFuncSetAttribute(latent_expand_kernel<TI, T, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                                 static_cast<int>(smem)) != cudaSuccess) return -3;                     \
    launch_k(latent_expand_kernel<TI, T, R>, grid, dim3(256), smem, STREAM, part_o, part_ml, splits, (const T*)w_uv, ldw, \
             (const TI*)gate, gate_ld, (T*)out, out_ld, B, H, rank, vdim);                                              \
  }
#define GO(TI, T)                        \
  {                                      \
    if (rows == 8) GO2(TI, T, 8)         \
    else if (rows == 4) GO2(TI, T, 4)    \
    else GO2(TI, T, 1)                   \
  }
  if (f32) GO(float, float)
  else if (in_f32) GO(float, bf16_t)
  else GO(bf16_t, bf16_t)
#undef GO
#undef GO2
  return DONE;
}

template <typename TI, typename T>
static void launch_rms_residual(void* a, int ld_a, int clear, const float* bias, const float* w, float* x, void* xb, int ld_xb,
                                int rows, int E, float eps, float mult, float* zero, int nzero, cudaStream_t st) {
  const int nv = (E % 8 == 0 && ld_a % 8 == 0 && ld_xb % 8 == 0) ? (E / 8 + 255) / 256 : 0;
  const bool aligned = !((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(xb) |
                          reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(bias)) & 15);
#define GO(NV)                                                                                                        \
  launch_k(rms_residual_vec_kernel<TI, T, NV>, dim3(rows), dim3(256), 0, st, (TI*)a, ld_a, clear, bias, w, x, (T*)xb, ld_xb, E, \
           eps, mult, zero, nzero)
  if (aligned && nv == 1) GO(1);
  else if (aligned && nv == 2) GO(2);
  else if (aligned && nv == 3) GO(3);
  else if (aligned && nv == 4) GO(4);
  else
    launch_k(rms_residual_kernel<TI, T>, dim3(rows), dim3(256), 0, st, (TI*)a, ld_a, clear, bias, w, x, (T*)xb, ld_xb, E, eps, mult,
             zero, nzero);
#undef GO
}

B200_API int b200_rms_residual(void* a, int ld_a, int in_f32, int clear, const float* bias, const float* w, float* x, void* xb,
                               int ld_xb, int rows, int E, float eps, float mult, float* zero, int nzero, int f32, void* stream) {
  if (rows <= 0 || E <= 0 || (clear && !in_f32) || (f32 && !in_f32) || (nzero && !zero)) return -1;
  if (f32) launch_rms_residual<float, float>(a, ld_a, clear, bias, w, x, xb, ld_xb, rows, E, eps, mult, zero, nzero, STREAM);
  else if (in_f32) launch_rms_residual<float, bf16_t>(a, ld_a, clear, bias, w, x, xb, ld_xb, rows, E, eps, mult, zero, nzero, STREAM);
  else launch_rms_residual<bf16_t, bf16_t>(a, ld_a, clear, bias, w, x, xb, ld_xb, rows, E, eps, mult, zero, nzero, STREAM);
  return DONE;
}

B200_API int b200_rmsnorm_rows(const float* x, const int* idx, const float* w, void* y, int ld_y, int rows, int E, float eps, float w_add,
                               float mult, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (f32) launch_k(rmsnorm_rows_kernel<float>, dim3(rows), dim3(256), 0, STREAM, x, idx, w, (float*)y, ld_y, E, eps, w_add, mult);
  else launch_k(rmsnorm_rows_kernel<bf16_t>, dim3(rows), dim3(256), 0, STREAM, x, idx, w, (bf16_t*)y, ld_y, E, eps, w_add, mult);
  return DONE;
}

B200_API int b200_bias_act(void* a, int ld_a, int in_f32, int clear, const float* bias, void* y, int ld_y, int rows, int N, int act,
                           int f32, void* stream) {
  if (rows <= 0 || rows > 65535 || N <= 0 || (clear && !in_f32) || (f32 && !in_f32)) return -1;
  const dim3 grid((N + 255) / 256, rows);
  if (f32) launch_k(bias_act_kernel<float, float>, grid, dim3(256), 0, STREAM, (float*)a, ld_a, clear, bias, (float*)y, ld_y, N, act);
  else if (in_f32) launch_k(bias_act_kernel<float, bf16_t>, grid, dim3(256), 0, STREAM, (float*)a, ld_a, clear, bias, (bf16_t*)y, ld_y, N, act);
  else launch_k(bias_act_kernel<bf16_t, bf16_t>, grid, dim3(256), 0, STREAM, (bf16_t*)a, ld_a, clear, bias, (bf16_t*)y, ld_y, N, act);
  return DONE;
}

B200_API int b200_sgemm_tile_rows() { return SG; }

B200_API int b200_sgemm_nt(const float* A, const float* B, const float* bias, float* C, int M, int N, int K, int lda, int ldb, int ldc,
                           int act, int act_lo, int act_hi, const int* group, const int* n_tiles, void* stream) {
  if (M <= 0 || N <= 0 || K <= 0 || (N + SG - 1) / SG > 65535 || !group != !n_tiles) return -1;
  sgemm_nt_kernel<<<dim3((M + SG - 1) / SG, (N + SG - 1) / SG), 256, 0, STREAM>>>(A, B, bias, C, M, N, K, lda, ldb, ldc, act, act_lo, act_hi,
                                                                                                    group, n_tiles);
  return DONE;
}
