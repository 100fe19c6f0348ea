// Kernels of grouped-query attention layers around their attention tiles:
//   * qkv_prep         : one projection row [q | k | v]: norm over all of q and of k, rotation of the leading dimensions of every
//                        head (halves paired), values mixed with those of another layer; keys and values go to the step's key
//                        stream and to the ring of the sequence
//   * qkv_heads        : the same for layers that norm every head of q and k (after the rotation) and of v by itself
//   * attention_merge  : key splits of a decode step, with an optional sink in the softmax's denominator
// Storage types: bf16 (serving) or fp32; arithmetic is fp32.  This file is built without fast-math approximations.
#include "rowops.cuh"

namespace b200 {

struct QkvRow {
  int ld_in, off_k, off_v;        // projection row, q at column 0
  int H, G, dim, vdim, rot;       // rot: rotated dimensions of a head (0: none)
  int ld_q, ld_kv, kv_v;          // q row; key / value row: k at 0, v at kv_v
  int cap, ld_first, ld_fout;     // ring slots of a sequence; pitches of the values mixed in / kept
  float eps;
  const float *q_norm, *k_norm;   // null: no norm
  const float *cosT, *sinT;       // [positions, rot / 2]
  const float* lam;               // value mixing: v = (1 - lam) v + lam first; null: none
  const int *pos, *row;
  const int *sidx, *end;          // stream index; position after the portion's last token (null: every token goes to the ring)
  int keep;                       // the ring holds the first `keep` positions of a sequence for good
  const float* bias;              // of the projection row (null: none, or added already)
};

// The ring row of position p of token t, or null when it is not kept.
template <typename T>
__device__ __forceinline__ T* ring_row(const QkvRow& P, T* cache, size_t t, int p) {
  if (!cache || (P.end && p >= P.keep && p < P.end[t] - (P.cap - P.keep))) return nullptr;
  return cache + (static_cast<size_t>(P.row[t]) * P.cap + ring_slot(p, P.cap, P.keep)) * P.ld_kv;
}

template <int W> struct Pack { float v[W]; };
template <int W, typename T> __device__ __forceinline__ Pack<W> ldw(const T* p) {
  Pack<W> r;
  if constexpr (W == 8) ld8(p, r.v);
  else r.v[0] = ldf(p);
  return r;
}
template <int W, typename T> __device__ __forceinline__ void stw(T* p, const Pack<W>& r) {
  if constexpr (W == 8) st8(p, r.v);
  else stf(p, r.v[0]);
}

// One CTA per token, W columns per access.  q may lie in the projection row itself: a pair of halves is read and written by one
// thread.
template <typename TI, typename T, typename TF, int W>
__global__ void __launch_bounds__(128)
qkv_prep_kernel(const TI* in, T* q, const TF* __restrict__ first, float* __restrict__ first_out, T* __restrict__ cache,
                T* __restrict__ stream, const QkvRow P) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const size_t t = blockIdx.x;
  const TI* r = in + t * P.ld_in;
  const int p = P.pos[t];
  T* qd = q + t * P.ld_q;
  T* kc = ring_row(P, cache, t, p);
  T* ks = stream ? stream + static_cast<size_t>(P.sidx[t]) * P.ld_kv : nullptr;
  float rq = 1.f, rk = 1.f;
  if (P.q_norm) {
    const int nq = P.H * P.dim, nk = P.G * P.dim;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x * W; i < nq + nk; i += 128 * W) {
      const bool isq = i < nq;
      const Pack<W> a = ldw<W>(isq ? r + i : r + P.off_k + (i - nq));
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < W; ++j) s += a.v[j] * a.v[j];
      if (isq) sq += s;
      else sk += s;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) {
      red[threadIdx.x >> 5] = sq;
      red[4 + (threadIdx.x >> 5)] = sk;
    }
    __syncthreads();
    rq = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / static_cast<float>(nq) + P.eps);
    rk = 1.f / sqrtf((red[4] + red[5] + red[6] + red[7]) / static_cast<float>(nk) + P.eps);
  }
  const int half = P.rot >> 1, pairs = half / W, units = pairs + (P.dim - P.rot) / W;   // pairs of packs, then packs that stay
  const float* ct = P.cosT + static_cast<size_t>(p) * half;
  const float* st = P.sinT + static_cast<size_t>(p) * half;
  for (int u = threadIdx.x; u < (P.H + P.G) * units; u += 128) {
    const int h = u / units, c = u - h * units;
    const bool isq = h < P.H;
    const int at = (isq ? h : h - P.H) * P.dim;
    const TI* src = r + (isq ? at : P.off_k + at);
    const float* nw = isq ? P.q_norm : P.k_norm;
    const float rs = isq ? rq : rk;
    const int i0 = c < pairs ? c * W : P.rot + (c - pairs) * W, i1 = i0 + half;
    Pack<W> a = ldw<W>(src + i0), b;
    if (c < pairs) b = ldw<W>(src + i1);
    if (nw) {
      const Pack<W> wa = ldw<W>(nw + at + i0);
#pragma unroll
      for (int j = 0; j < W; ++j) a.v[j] *= rs * wa.v[j];
      if (c < pairs) {
        const Pack<W> wb = ldw<W>(nw + at + i1);
#pragma unroll
        for (int j = 0; j < W; ++j) b.v[j] *= rs * wb.v[j];
      }
    }
    if (c < pairs) {
      const Pack<W> cs = ldw<W>(ct + i0), sn = ldw<W>(st + i0);
#pragma unroll
      for (int j = 0; j < W; ++j) {
        const float x = a.v[j], y = b.v[j];
        a.v[j] = x * cs.v[j] - y * sn.v[j];
        b.v[j] = y * cs.v[j] + x * sn.v[j];
      }
    }
    if (isq) {
      stw<W>(qd + at + i0, a);
      if (c < pairs) stw<W>(qd + at + i1, b);
    } else {
      if (kc) {
        stw<W>(kc + at + i0, a);
        if (c < pairs) stw<W>(kc + at + i1, b);
      }
      if (ks) {
        stw<W>(ks + at + i0, a);
        if (c < pairs) stw<W>(ks + at + i1, b);
      }
    }
  }
  const float lam = P.lam ? *P.lam : 0.f;
  for (int i = threadIdx.x * W; i < P.G * P.vdim; i += 128 * W) {
    Pack<W> v = ldw<W>(r + P.off_v + i);
    if (first_out) stw<W>(first_out + t * P.ld_fout + i, v);
    if (P.lam) {
      const Pack<W> f = ldw<W>(first + t * P.ld_first + i);
#pragma unroll
      for (int j = 0; j < W; ++j) v.v[j] = (1.f - lam) * v.v[j] + lam * f.v[j];
    }
    if (kc) stw<W>(kc + P.kv_v + i, v);
    if (ks) stw<W>(ks + P.kv_v + i, v);
  }
}

// LANES lanes per (token, head of q, k or v): one pass for the sum of squares, which a rotation leaves alone, and one for the result (ONE:
// a head is at most one unit per lane and is read once).  q may lie in the projection row itself.
template <typename TI, typename T, int W, int LANES, bool ONE>
__global__ void __launch_bounds__(128)
qkv_heads_kernel(const TI* in, T* q, T* __restrict__ cache, T* __restrict__ stream, const QkvRow P, int total) {
  pdl_trigger();
  pdl_wait();
  const int heads = P.H + 2 * P.G, id = blockIdx.x * (128 / LANES) + threadIdx.x / LANES, lane = threadIdx.x % LANES;
  const bool on = id < total;                                   // every lane takes part in the sums
  const size_t t = on ? id / heads : 0;
  const int h = on ? id % heads : 0, p = P.pos[t];
  const int kind = h < P.H ? 0 : h < P.H + P.G ? 1 : 2, hh = kind == 0 ? h : kind == 1 ? h - P.H : h - P.H - P.G;
  const int n = kind == 2 ? P.vdim : P.dim, at = hh * n, col = (kind == 0 ? 0 : kind == 1 ? P.off_k : P.off_v) + at;
  const TI* src = in + t * P.ld_in + col;
  const float* bias = P.bias ? P.bias + col : nullptr;
  auto load = [&](int i) {
    Pack<W> a = ldw<W>(src + i);
    if (bias) {
      const Pack<W> b = ldw<W>(bias + i);
#pragma unroll
      for (int j = 0; j < W; ++j) a.v[j] += b.v[j];
    }
    return a;
  };
  const int half = kind == 2 ? 0 : P.rot >> 1, pairs = half / W, units = pairs + (n - 2 * half) / W;
  const float* ct = P.cosT + static_cast<size_t>(p) * half;
  const float* st = P.sinT + static_cast<size_t>(p) * half;
  auto first = [&](int c) { return c < pairs ? c * W : 2 * half + (c - pairs) * W; };
  float ss = 0.f;
  Pack<W> one_a, one_b;
  if constexpr (ONE) {
    if (lane < units) {
      one_a = load(first(lane));
#pragma unroll
      for (int j = 0; j < W; ++j) ss += one_a.v[j] * one_a.v[j];
      if (lane < pairs) {
        one_b = load(first(lane) + half);
#pragma unroll
        for (int j = 0; j < W; ++j) ss += one_b.v[j] * one_b.v[j];
      }
    }
  } else {
    for (int i = lane * W; i < n; i += LANES * W) {
      const Pack<W> a = load(i);
#pragma unroll
      for (int j = 0; j < W; ++j) ss += a.v[j] * a.v[j];
    }
  }
#pragma unroll
  for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!on) return;
  const float f = 1.f / sqrtf(ss / static_cast<float>(n) + P.eps);
  T* dst[2] = {nullptr, nullptr};
  if (kind == 0) {
    dst[0] = q + t * P.ld_q + at;
  } else {
    const int off = (kind == 2 ? P.kv_v : 0) + at;
    if (T* kc = ring_row(P, cache, t, p)) dst[0] = kc + off;
    if (stream) dst[1] = stream + static_cast<size_t>(P.sidx[t]) * P.ld_kv + off;
  }
  for (int c = lane; c < units; c += LANES) {
    const int i0 = first(c), i1 = i0 + half;
    Pack<W> a = ONE ? one_a : load(i0), b;
#pragma unroll
    for (int j = 0; j < W; ++j) a.v[j] *= f;
    if (c < pairs) {
      b = ONE ? one_b : load(i1);
      const Pack<W> cs = ldw<W>(ct + i0), sn = ldw<W>(st + i0);
#pragma unroll
      for (int j = 0; j < W; ++j) {
        const float x = a.v[j], y = b.v[j] * f;
        a.v[j] = x * cs.v[j] - y * sn.v[j];
        b.v[j] = y * cs.v[j] + x * sn.v[j];
      }
    }
#pragma unroll
    for (int k = 0; k < 2; ++k)
      if (dst[k]) {
        stw<W>(dst[k] + i0, a);
        if (c < pairs) stw<W>(dst[k] + i1, b);
      }
  }
}

// out[b, h * vdim + d] = sum over splits / (sum of the softmax + exp(sink)).  CTA per (sequence, head): every warp takes each fourth
// split, all its pieces requested at once.
template <typename T>
__global__ void __launch_bounds__(128)
attention_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, const float* __restrict__ sink,
                       T* __restrict__ out, int ld_out, int H, int vdim, int splits) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sums[];                               // [4][vdim padded to four]
  const int i = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = i / H, h = i - b * H, vs = (vdim + 7) & ~7, v4 = (vdim + 3) & ~3;
  const float2 e = lane < splits ? *reinterpret_cast<const float2*>(part_ml + (static_cast<size_t>(i) * splits + lane) * 2)
                                 : make_float2(-INFINITY, 0.f);
  const float sk = sink ? sink[h] : -INFINITY;
  const float m = fmaxf(warp_max(e.x), sk);
  const float w = e.x == -INFINITY ? 0.f : expf(e.x - m);
  const float mine = w / (warp_sum(w * e.y) + (sink ? expf(sk - m) : 0.f));
  float f[8];
#pragma unroll
  for (int u = 0; u < 8; ++u) f[u] = __shfl_sync(0xffffffffu, mine, warp + 4 * u);   // zero past the splits
  const float* p = part_o + static_cast<size_t>(i) * splits * vs;
  for (int d = 4 * lane; d < v4; d += 128) {
    float x[8][4];
#pragma unroll
    for (int u = 0; u < 8; ++u)
      if (f[u] != 0.f) ld4(p + static_cast<size_t>(warp + 4 * u) * vs + d, x[u]);    // an empty split's partial is not initialised
    float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int u = 0; u < 8; ++u)
#pragma unroll
      for (int k = 0; k < 4; ++k) o[k] += f[u] != 0.f ? f[u] * x[u][k] : 0.f;
    *reinterpret_cast<float4*>(sums + warp * v4 + d) = make_float4(o[0], o[1], o[2], o[3]);
  }
  __syncthreads();
  for (int d = threadIdx.x; d < vdim; d += 128)
    stf(out + static_cast<size_t>(b) * ld_out + h * vdim + d, sums[d] + sums[v4 + d] + sums[2 * v4 + d] + sums[3 * v4 + d]);
}

}  // namespace b200

using namespace b200;
typedef __nv_bfloat16 bf16_t;
#define STREAM reinterpret_cast<cudaStream_t>(stream)
#define DONE (cudaGetLastError() == cudaSuccess ? 0 : -2)

static bool row_ok(const QkvRow& P, int T, const void* cache, const void* stream_buf, int in_f32, int f32) {
  return T > 0 && P.H > 0 && P.G > 0 && P.H % P.G == 0 && P.dim > 0 && P.vdim > 0 && P.rot >= 0 && !(P.rot & 1) && P.rot <= P.dim && P.cap > 0 && P.keep >= 0 &&
         P.pos && (!cache || P.row) && (!stream_buf || P.sidx) && (!P.rot || (P.cosT && P.sinT)) && (!f32 || in_f32);
}

// in: T projection rows (fp32 accumulators with in_f32); q: destination of the queries (may be `in`); first: values of the layer
// that provides them (fp32 with first_f32), first_out: fp32 copy of this layer's unmixed values; stream_buf / cache may be null.
B200_API int b200_qkv_prep(const void* in, void* q, const void* first, float* first_out, void* cache, void* stream_buf, const QkvRow* Pp,
                           int T, int in_f32, int f32, int first_f32, void* stream) {
  const QkvRow P = *Pp;
  if (!row_ok(P, T, cache, stream_buf, in_f32, f32) || (P.lam && !first) || (!P.q_norm != !P.k_norm) || P.bias) return -1;
  const uintptr_t addr = reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(first) |
                         reinterpret_cast<uintptr_t>(first_out) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(stream_buf) |
                         reinterpret_cast<uintptr_t>(P.q_norm) | reinterpret_cast<uintptr_t>(P.k_norm) | reinterpret_cast<uintptr_t>(P.cosT) |
                         reinterpret_cast<uintptr_t>(P.sinT);
  const bool vec = !(addr & 15) && !((P.dim | (P.rot >> 1) | (P.G * P.vdim) | P.ld_in | P.off_k | P.off_v | P.ld_q | P.ld_kv | P.kv_v | P.ld_first | P.ld_fout) & 7);
#define GO2(TI, T_, TF, W) \
  launch_k(qkv_prep_kernel<TI, T_, TF, W>, dim3(T), dim3(128), 0, STREAM, (const TI*)in, (T_*)q, (const TF*)first, first_out, (T_*)cache, (T_*)stream_buf, P)
#define GO(TI, T_, TF) { if (vec) GO2(TI, T_, TF, 8); else GO2(TI, T_, TF, 1); }
  if (f32) GO(float, float, float)
  else if (in_f32) GO(float, bf16_t, float)
  else if (first_f32) GO(bf16_t, bf16_t, float)
  else GO(bf16_t, bf16_t, bf16_t)
#undef GO
#undef GO2
  return DONE;
}

// Arguments as in b200_qkv_prep; neither weighted norms nor value mixing.
B200_API int b200_qkv_heads(const void* in, void* q, void* cache, void* stream_buf, const QkvRow* Pp, int T, int in_f32, int f32, void* stream) {
  const QkvRow P = *Pp;
  const long long total = static_cast<long long>(T) * (P.H + 2 * P.G);
  if (!row_ok(P, T, cache, stream_buf, in_f32, f32) || P.q_norm || P.lam || total > 0x7fffffffll - 128) return -1;
  const uintptr_t addr = reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(stream_buf) |
                         reinterpret_cast<uintptr_t>(P.cosT) | reinterpret_cast<uintptr_t>(P.sinT) | reinterpret_cast<uintptr_t>(P.bias);
  const bool vec = !(addr & 15) && !((P.dim | (P.rot >> 1) | P.vdim | P.ld_in | P.off_k | P.off_v | P.ld_q | P.ld_kv | P.kv_v) & 7);
  const int n = P.dim > P.vdim ? P.dim : P.vdim;
#define GO2(TI, T_, W, LN, ONE) \
  launch_k(qkv_heads_kernel<TI, T_, W, LN, ONE>, dim3(static_cast<unsigned>((total + 128 / LN - 1) / (128 / LN))), dim3(128), 0, STREAM, (const TI*)in, (T_*)q, (T_*)cache, (T_*)stream_buf, P, static_cast<int>(total))
#define GO(TI, T_) { if (!vec) GO2(TI, T_, 1, 32, false); else if (n <= 64) GO2(TI, T_, 8, 8, true); else if (n <= 128) GO2(TI, T_, 8, 16, true); else if (n <= 256) GO2(TI, T_, 8, 32, true); else GO2(TI, T_, 8, 32, false); }
  if (f32) GO(float, float)
  else if (in_f32) GO(float, bf16_t)
  else GO(bf16_t, bf16_t)
#undef GO
#undef GO2
  return DONE;
}

B200_API int b200_attention_merge(const float* part_o, const float* part_ml, const float* sink, void* out, int ld_out, int B, int H, int vdim,
                                  int splits, int f32, void* stream) {
  if (B <= 0 || H <= 0 || vdim <= 0 || splits < 1 || splits > 32) return -1;
  const size_t smem = 4 * ((vdim + 3) & ~3) * sizeof(float);
  if (smem > 48 * 1024 || static_cast<long long>(B) * H > 0x7fffffffll) return -1;
  if (f32) launch_k(attention_merge_kernel<float>, dim3(B * H), dim3(128), smem, STREAM, part_o, part_ml, sink, (float*)out, ld_out, H, vdim, splits);
  else launch_k(attention_merge_kernel<bf16_t>, dim3(B * H), dim3(128), smem, STREAM, part_o, part_ml, sink, (bf16_t*)out, ld_out, H, vdim, splits);
  return DONE;
}
