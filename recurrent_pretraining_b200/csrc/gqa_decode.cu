// Decode attention of grouped-query layers: one new token per sequence against its cached keys and values, bf16 matrix units,
// fp32 softmax.  Either with a learned distance bias over all cached positions, or (RING) capped scores over the window or the
// chunk that the sequence's ring holds.  A decode step is bound by the stream of keys and values, so one warp owns 16
// keys at a time for all heads of a group (padded to the 16 rows of an MMA) and every byte is read once.
//
// CTA per (key split, key / value head, sequence), four warps: a warp takes every fourth 16-key tile of the split, staged by
// cp.async in a ring of its own (no barriers in the loop), and keeps its own running softmax; the warps are joined in shared
// memory at the end.  The new token's key and value are not in the cache yet: the warp that meets its position forms them
// from the projection row and appends them.
//
// RING: position p lies in slot p % cap.  Queries and the new key are normed over the whole projection and / or rotated, the new
// value is mixed with another layer's where they are formed; or every head is normed by itself (q and k once rotated, v).  Under a window
// the sequence's first `keep` positions may stay visible: they have the ring's first slots for good and are counted in front of the
// window's keys.  Bounded scores need no running maximum.  With a single split the sink and the division are applied here.
#include "rowops.cuh"
#include "softmax_math.cuh"

namespace b200 {

struct GqaDecode {
  int H, G, dim, vdim, ld_in, off_k, off_v;        // columns of the projection row (q at 0)
  int ld_kv, kv_v, cap;                            // cache [rows, cap, ld_kv]: k at 0, v at kv_v
  int splits, bias_len, ld_bias, bias_lead;
  int temp_every;
  float temp_coef, scale;
  const float* in_bias;                            // bias of the raw projection row
  const float* bias;                               // [H, ld_bias] in log2 units, distance d at bias_lead + d
  const int *pos, *row;
  __nv_bfloat16* cache;
  float* part_o;                                   // [B, H, splits, vdim padded to eight], unnormalised
  float* part_ml;                                  // [B, H, splits, 2] (max in natural-log units, sum)
  // RING
  int size, chunked;                               // visible: the last `size` positions, or the chunk of `size` positions
  int rot, ld_first, ld_fout, ld_out;
  float eps, softcap;                              // softcap 0: scores are not capped
  const float *q_norm, *k_norm, *cosT, *sinT;      // null: no norm; tables [positions, rot / 2]
  const float *lam, *first;                        // value mixing: (1 - lam) v + lam first [B, ld_first]; null: none
  float* first_out;                                // [B, ld_fout] unmixed values; null: not wanted
  const float* sink;                               // [H]; null: none
  __nv_bfloat16* out;                              // [B, ld_out] with a single split, else null
  int keep, head_norm;                             // kept first positions; every head of q, k and v is normed without weights
  float bound;                                     // no score is larger (0: not known)
};

constexpr int GD_KEYS = 16, GD_WARPS = 4;

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Row pitches in bytes of staged q / k and v rows: whole 16-column steps and 16 bytes more, so that the eight rows of an
// ldmatrix fall into different banks.
__host__ __device__ constexpr int gd_pitch(int cols) { return ((cols + 15) & ~15) * 2 + 16; }

// Entry i of a head with bias (null: none), scaled by r and the weights w (null: none) and rotated (halves paired).
template <typename TI>
__device__ __forceinline__ float head_entry(const TI* x, int i, const float* bias, const float* w, float r, int rot, const float* ct, const float* st) {
  auto entry = [&](int e) { return (ldf(x + e) + (bias ? bias[e] : 0.f)) * (w ? r * w[e] : r); };
  float v = entry(i);
  if (i < rot) {
    const int half = rot >> 1, j = i < half ? i : i - half, o = i < half ? i + half : i - half;
    const float u = entry(o);
    v = i < half ? v * ct[j] - u * st[j] : v * ct[j] + u * st[j];
  }
  return v;
}

// Eight entries from i (a multiple of eight) on.
template <typename TI>
__device__ __forceinline__ void head_entries8(const TI* x, int i, const float* bias, const float* w, float r, int rot, const float* ct, const float* st, float (&v)[8]) {
  const int half = rot >> 1;
  if (i < rot && (half & 7)) {                                         // pairs do not fall into the same places of two groups
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = head_entry(x, i + j, bias, w, r, rot, ct, st);
    return;
  }
  auto entries = [&](int e, float (&y)[8]) {
    ld8(x + e, y);
    float f[8];
    if (bias) {
      ld8(bias + e, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) y[j] += f[j];
    }
    if (w) ld8(w + e, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) y[j] *= w ? r * f[j] : r;
  };
  entries(i, v);
  if (i < rot) {
    const bool low = i < half;
    const int c = low ? i : i - half, o = low ? i + half : i - half;
    float u[8], cs[8], sn[8];
    entries(o, u);
    ld8(ct + c, cs);
    ld8(st + c, sn);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = low ? v[j] * cs[j] - u[j] * sn[j] : v[j] * cs[j] + u[j] * sn[j];
  }
}

// NV: 16-column steps of the values that the accumulators hold.
// HEADS (with RING): kept positions, biases, heads normed by themselves.
template <typename TI, int NV, int STAGES, bool RING, bool HEADS>
__global__ void __launch_bounds__(128)
gqa_decode_kernel(const TI* __restrict__ in, const GqaDecode P) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, b = blockIdx.z;
  const int group = P.H / P.G, chunks = (group + 15) / 16;
  const int g = blockIdx.y / chunks, h0 = g * group + (blockIdx.y % chunks) * 16, nh = min(16, (g + 1) * group - h0);
  const int pos = P.pos[b];
  const int key_first = RING ? (P.chunked ? pos - pos % P.size : max(0, pos - P.size + 1)) : 0;
  const int keep = HEADS ? P.keep : 0, kept = HEADS ? min(keep, key_first) : 0;                  // keys are counted: kept ones in front of the window, then the window
  const int newest = kept + pos - key_first, nkeys = newest + 1;
  const int slot0 = RING ? ring_slot(key_first, P.cap, keep) - kept : 0;
  auto slot_of = [&](int j) {
    if (HEADS && j < kept) return j;
    int s = slot0 + j;
    if (RING && s >= P.cap) s -= P.cap - keep;
    return s;
  };
  const int tiles = (nkeys + GD_KEYS - 1) / GD_KEYS, per = (tiles + P.splits - 1) / P.splits;
  const int tile0 = split * per, tile1 = min(tiles, tile0 + per);
  const int vs = (P.vdim + 7) & ~7;
  if (tile0 >= tile1) {                                                // not with a single split
    if (threadIdx.x < nh) {
      float* ml = P.part_ml + ((static_cast<size_t>(b) * P.H + h0 + threadIdx.x) * P.splits + split) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.f;
    }
    return;
  }
  const int kp = gd_pitch(P.dim), vp = gd_pitch(P.vdim);
  const int stage_bytes = GD_KEYS * (kp + vp);
  uint8_t* sq = smem;                                                  // [16][kp]
  uint8_t* ring = sq + 16 * kp + warp * STAGES * stage_bytes;
  const TI* r = in + static_cast<size_t>(b) * P.ld_in;
  __nv_bfloat16* base = P.cache + static_cast<size_t>(P.row[b]) * P.cap * P.ld_kv;
  // 16-byte pieces of a key row and a value row: a power of two of lanes per key, or several passes of 32
  const int kch = P.dim >> 3, ch = kch + (P.vdim >> 3);
  int lpk = 1;
  while (lpk < ch && lpk < 32) lpk <<= 1;
  const int kpp = 32 / lpk, lj = lane / lpk, lc = lane % lpk;          // keys per pass, this lane's key and first piece
  auto request = [&](int tile, int st) {
    const uint32_t s = smem_u32(ring + st * stage_bytes);
    const int last = max(newest - 1, 0), j0 = tile * GD_KEYS;          // keys past the newest repeat one that exists; they are masked
    const bool plain = j0 + GD_KEYS - 1 <= last && slot_of(j0 + GD_KEYS - 1) - slot_of(j0) == GD_KEYS - 1 && (!HEADS || j0 >= kept || j0 + GD_KEYS <= kept);
    const __nv_bfloat16* row0 = base + static_cast<size_t>(slot_of(min(j0, last)) + lj) * P.ld_kv;
    for (int c = lc; c < ch; c += lpk) {
      const bool isk = c < kch;
      const int at = isk ? g * P.dim + 8 * c : P.kv_v + g * P.vdim + 8 * (c - kch);
      const uint32_t dst = s + (isk ? 16 * c : GD_KEYS * kp + 16 * (c - kch));
      const int pitch = isk ? kp : vp;
      if (plain) {                                                     // neighbouring slots
        const __nv_bfloat16* src = row0 + at;
        const size_t step = static_cast<size_t>(kpp) * P.ld_kv;
#pragma unroll 8
        for (int j = lj; j < GD_KEYS; j += kpp, src += step) cp_async16(dst + j * pitch, src);
      } else {
#pragma unroll 4
        for (int j = lj; j < GD_KEYS; j += kpp) cp_async16(dst + j * pitch, base + at + static_cast<size_t>(slot_of(min(j0 + j, last))) * P.ld_kv);
      }
    }
  };
  const int first = tile0 + warp;
  const int mine = first < tile1 ? (tile1 - 1 - first) / GD_WARPS + 1 : 0;
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) {
    if (s < mine) request(first + s * GD_WARPS, s);
    cp_commit();
  }
  float rq = 1.f, rk = 1.f;
  const float *cos_t = nullptr, *sin_t = nullptr;
  __shared__ float rh[18];                                             // factors of the heads' own norms: q heads, then k and v
  if constexpr (RING) {
    if (HEADS && P.head_norm) {                                                 // a rotation leaves the sum of squares alone
      for (int i = warp; i < nh + 2; i += GD_WARPS) {
        const int n = i <= nh ? P.dim : P.vdim, col = i < nh ? (h0 + i) * P.dim : i == nh ? P.off_k + g * P.dim : P.off_v + g * P.vdim;
        float t = 0.f;
        for (int c = 8 * lane; c < n; c += 256) {
          float v[8];
          head_entries8(r + col, c, P.in_bias ? P.in_bias + col : nullptr, nullptr, 1.f, 0, nullptr, nullptr, v);
#pragma unroll
          for (int j = 0; j < 8; ++j) t += v[j] * v[j];
        }
        t = warp_sum(t);
        if (lane == 0) rh[i] = 1.f / sqrtf(t / static_cast<float>(n) + P.eps);
      }
      __syncthreads();
      rk = rh[nh];
    }
    cos_t = P.cosT + static_cast<size_t>(pos) * (P.rot >> 1);
    sin_t = P.sinT + static_cast<size_t>(pos) * (P.rot >> 1);
    if (P.q_norm) {
      __shared__ float red[8];
      const int nq = P.H * P.dim, nk = P.G * P.dim;                    // multiples of eight
      float sq = 0.f, sk = 0.f;
#pragma unroll 4
      for (int i = 8 * threadIdx.x; i < nq + nk; i += 1024) {
        float v[8], t = 0.f;
        ld8(i < nq ? r + i : r + P.off_k + (i - nq), v);
#pragma unroll
        for (int j = 0; j < 8; ++j) t += v[j] * v[j];
        if (i < nq) sq += t;
        else sk += t;
      }
      sq = warp_sum(sq);
      sk = warp_sum(sk);
      if (lane == 0) {
        red[warp] = sq;
        red[4 + warp] = sk;
      }
      __syncthreads();
      rq = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / static_cast<float>(nq) + P.eps);
      rk = 1.f / sqrtf((red[4] + red[5] + red[6] + red[7]) / static_cast<float>(nk) + P.eps);
    }
  }
  // queries, zero in the padding rows and columns; the ring's padding columns are zeroed once
  if constexpr (RING) {
    const int vecs = kp / 16;                                          // groups of eight columns of a staged row
    for (int i = threadIdx.x; i < 16 * vecs; i += 128) {
      const int hh = i / vecs, c = 8 * (i - hh * vecs);
      float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (hh < nh && c < P.dim) {
        const int at = (h0 + hh) * P.dim;
        head_entries8(r + at, c, HEADS && P.in_bias ? P.in_bias + at : nullptr, P.q_norm ? P.q_norm + at : nullptr, HEADS && P.head_norm ? rh[hh] : rq, P.rot, cos_t, sin_t, v);
      }
      st8(reinterpret_cast<__nv_bfloat16*>(sq) + hh * (kp / 2) + c, v);
    }
  } else {
    for (int i = threadIdx.x; i < 16 * (kp / 2); i += 128) {
      const int hh = i / (kp / 2), c = i - hh * (kp / 2);
      float v = 0.f;
      if (hh < nh && c < P.dim) v = ldf(r + (h0 + hh) * P.dim + c) + P.in_bias[(h0 + hh) * P.dim + c];
      reinterpret_cast<__nv_bfloat16*>(sq)[i] = f2bf(v);
    }
  }
  for (int i = lane; i < STAGES * GD_KEYS; i += 32) {
    uint8_t* s = ring + (i / GD_KEYS) * stage_bytes;
    __nv_bfloat16* kr = reinterpret_cast<__nv_bfloat16*>(s + (i % GD_KEYS) * kp);
    __nv_bfloat16* vr = reinterpret_cast<__nv_bfloat16*>(s + GD_KEYS * kp + (i % GD_KEYS) * vp);
    for (int c = P.dim; c < kp / 2; ++c) kr[c] = f2bf(0.f);
    for (int c = P.vdim; c < vp / 2; ++c) vr[c] = f2bf(0.f);
  }
  __syncthreads();
  // rows of this thread's accumulators: heads lane / 4 and lane / 4 + 8
  const int ra = lane >> 2;
  float rowmul = P.scale * 1.4426950408889634f;
  if (!RING && P.temp_every > 0) rowmul *= query_temperature(pos, P.temp_every, P.temp_coef);
  const float* bias_row[2] = {nullptr, nullptr};
  float bias_far[2] = {0.f, 0.f};
  const int far = P.bias_len - 1;
  if constexpr (!RING) {
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      bias_row[k] = P.bias + static_cast<size_t>(min(h0 + ra + 8 * k, P.H - 1)) * P.ld_bias + P.bias_lead;
      bias_far[k] = bias_row[k][far];
    }
  }
  const bool capped = RING && P.softcap > 0.f;
  const float cap_log2 = P.softcap * 1.4426950408889634f, cap_exp = capped ? 2.f * rowmul / P.softcap : 0.f;
  const bool bounded = RING && (capped ? cap_log2 <= 80.f : HEADS && P.bound > 0.f && P.bound * 1.4426950408889634f <= 80.f);      // weights lie in 2^(-80 .. 80): no running maximum
  const float m_start = bounded ? 0.f : -INFINITY;
  float m[2] = {m_start, m_start}, l[2] = {0.f, 0.f};
  float o[NV][2][4];
#pragma unroll
  for (int n = 0; n < NV; ++n)
#pragma unroll
    for (int k = 0; k < 2; ++k) o[n][k][0] = o[n][k][1] = o[n][k][2] = o[n][k][3] = 0.f;
  const int ksteps = (P.dim + 15) >> 4, vsteps = (P.vdim + 15) >> 4;
  // ldmatrix row / column of this lane: A (q) rows by lane & 15; B of k: keys (lane & 7) + 8 (lane >> 4), columns 8 ((lane >> 3) & 1);
  // B of v (transposed): keys lane & 15, columns 8 (lane >> 4)
  const uint32_t aq = smem_u32(sq) + (lane & 15) * kp + (lane >> 4) * 16;
  const uint32_t bk = ((lane & 7) + 8 * (lane >> 4)) * kp + ((lane >> 3) & 1) * 16;
  const uint32_t bv = GD_KEYS * kp + (lane & 15) * vp + (lane >> 4) * 16;
  for (int it = 0; it < mine; ++it) {
    const int st = it % STAGES, tile = first + it * GD_WARPS;
    cp_wait<STAGES - 2>();
    __syncwarp();
    {
      const int nx = it + STAGES - 1;
      if (nx < mine) request(first + nx * GD_WARPS, nx % STAGES);
      cp_commit();
    }
    uint8_t* sb = ring + st * stage_bytes;
    const int key0 = tile * GD_KEYS;
    if (key0 + GD_KEYS > newest) {                                     // the newest token lies in this tile
      const int j = newest - key0;
      __nv_bfloat16* dst = base + static_cast<size_t>(slot_of(newest)) * P.ld_kv;
      if constexpr (RING) {
        for (int c = 8 * lane; c < P.dim + P.vdim; c += 256) {
          const bool isk = c < P.dim;
          const int cc = isk ? c : c - P.dim, vc = g * P.vdim + cc;
          float f[8];
          if (isk) {
            head_entries8(r + P.off_k + g * P.dim, cc, HEADS && P.in_bias ? P.in_bias + P.off_k + g * P.dim : nullptr, P.k_norm ? P.k_norm + g * P.dim : nullptr, rk,
                          P.rot, cos_t, sin_t, f);
          } else {
            head_entries8(r + P.off_v + g * P.vdim, cc, HEADS && P.in_bias ? P.in_bias + P.off_v + g * P.vdim : nullptr, nullptr, HEADS && P.head_norm ? rh[nh + 1] : 1.f, 0,
                          nullptr, nullptr, f);
            if (P.first_out) st8(P.first_out + static_cast<size_t>(b) * P.ld_fout + vc, f);
            if (P.lam) {
              const float lam = *P.lam;
              float e[8];
              ld8(P.first + static_cast<size_t>(b) * P.ld_first + vc, e);
#pragma unroll
              for (int k = 0; k < 8; ++k) f[k] = (1.f - lam) * f[k] + lam * e[k];
            }
          }
          st8(reinterpret_cast<__nv_bfloat16*>(sb + (isk ? j * kp : GD_KEYS * kp + j * vp)) + cc, f);
          st8(dst + (isk ? g * P.dim : P.kv_v + g * P.vdim) + cc, f);
        }
      } else {
        for (int c = lane; c < P.dim + P.vdim; c += 32) {
          const bool isk = c < P.dim;
          const int cc = isk ? c : c - P.dim, col = isk ? P.off_k + g * P.dim + cc : P.off_v + g * P.vdim + cc;
          const __nv_bfloat16 v = f2bf(ldf(r + col) + P.in_bias[col]);
          reinterpret_cast<__nv_bfloat16*>(sb + (isk ? j * kp : GD_KEYS * kp + j * vp))[cc] = v;
          dst[(isk ? g * P.dim : P.kv_v + g * P.vdim) + cc] = v;
        }
      }
      __syncwarp();
    }
    const uint32_t s = smem_u32(sb);
    float c[2][4] = {};
#pragma unroll 4
    for (int t = 0; t < ksteps; ++t) {
      uint32_t a[4], k4[4];
      ldsm4(a, aq + 32 * t);
      ldsm4(k4, s + bk + 32 * t);
      mma_bf16(c[0], a, k4[0], k4[1]);
      mma_bf16(c[1], a, k4[2], k4[3]);
    }
    // c[n][0..1]: head ra, keys key0 + 8 n + 2 (lane & 3) + {0, 1}; c[n][2..3]: head ra + 8
    float p[2][4];
    float mx[2] = {-INFINITY, -INFINITY};
    if constexpr (RING) {
      const int d0 = newest - key0 - 2 * (lane & 3);
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = capped ? cap_log2 - 2.f * cap_log2 * rcp_approx(1.f + ex2_approx(c[n][e] * cap_exp)) : c[n][e] * rowmul;
          p[n][e] = d0 - 8 * n - (e & 1) >= 0 ? x : -INFINITY;
          mx[e >> 1] = fmaxf(mx[e >> 1], p[n][e]);
        }
    } else if (pos - key0 - (GD_KEYS - 1) >= far) {                           // every distance shares the last bucket
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          p[n][e] = fmaf(c[n][e], rowmul, bias_far[e >> 1]);
          mx[e >> 1] = fmaxf(mx[e >> 1], p[n][e]);
        }
    } else {
      const int d0 = pos - key0 - 2 * (lane & 3);
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = d0 - 8 * n - (e & 1);
          p[n][e] = d >= 0 ? fmaf(c[n][e], rowmul, bias_row[e >> 1][min(max(d, 0), far)]) : -INFINITY;
          mx[e >> 1] = fmaxf(mx[e >> 1], p[n][e]);
        }
    }
    float alpha[2] = {1.f, 1.f};
    bool moved = false;
    if (!bounded) {
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        mx[k] = fmaxf(mx[k], __shfl_xor_sync(0xffffffffu, mx[k], 1));
        mx[k] = fmaxf(mx[k], __shfl_xor_sync(0xffffffffu, mx[k], 2));
        const float mn = fmaxf(m[k], mx[k]);                             // finite: the tile's first key is visible
        alpha[k] = exp2f(m[k] - mn);
        moved |= mn != m[k];
        m[k] = mn;
        l[k] *= alpha[k];
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        p[n][e] = exp2f(p[n][e] - m[e >> 1]);
        l[e >> 1] += p[n][e];
      }
    if (!bounded && __any_sync(0xffffffffu, moved)) {
#pragma unroll
      for (int n = 0; n < NV; ++n)
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          o[n][k][0] *= alpha[0]; o[n][k][1] *= alpha[0];
          o[n][k][2] *= alpha[1]; o[n][k][3] *= alpha[1];
        }
    }
    const uint32_t pa[4] = {pack_bf16x2(p[0][0], p[0][1]), pack_bf16x2(p[0][2], p[0][3]), pack_bf16x2(p[1][0], p[1][1]), pack_bf16x2(p[1][2], p[1][3])};
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      if (n < vsteps) {
        uint32_t v4[4];
        ldsm4t(v4, s + bv + 32 * n);
#pragma unroll
        for (int k = 0; k < 2; ++k) mma_bf16(o[n][k], pa, v4[2 * k], v4[2 * k + 1]);
      }
    }
    __syncwarp();                                                      // the stage may be requested again
  }
  cp_wait<0>();
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    l[k] += __shfl_xor_sync(0xffffffffu, l[k], 1);
    l[k] += __shfl_xor_sync(0xffffffffu, l[k], 2);
  }
  // join the warps
  __syncthreads();
  float* sml = reinterpret_cast<float*>(smem);                         // [4][16][2]
  float* so = sml + GD_WARPS * 32;                                     // [4][16][vs]
  if ((lane & 3) == 0) {
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      sml[(warp * 16 + ra + 8 * k) * 2] = m[k];
      sml[(warp * 16 + ra + 8 * k) * 2 + 1] = l[k];
    }
  }
#pragma unroll
  for (int n = 0; n < NV; ++n)
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int col = 16 * n + 8 * k + 2 * (lane & 3);
      if (col < P.vdim) {
        *reinterpret_cast<float2*>(so + (warp * 16 + ra) * vs + col) = make_float2(o[n][k][0], o[n][k][1]);
        *reinterpret_cast<float2*>(so + (warp * 16 + ra + 8) * vs + col) = make_float2(o[n][k][2], o[n][k][3]);
      }
    }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * (P.vdim >> 2); i += 128) {
    const int hh = i / (P.vdim >> 2), col = 4 * (i - hh * (P.vdim >> 2));
    float mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < GD_WARPS; ++w) mm = fmaxf(mm, sml[(w * 16 + hh) * 2]);
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    float ll = 0.f;
#pragma unroll
    for (int w = 0; w < GD_WARPS; ++w) {
      const float f = exp2f(sml[(w * 16 + hh) * 2] - mm);
      const float4 x = *reinterpret_cast<const float4*>(so + (w * 16 + hh) * vs + col);
      v.x += f * x.x; v.y += f * x.y; v.z += f * x.z; v.w += f * x.w;
      ll += f * sml[(w * 16 + hh) * 2 + 1];
    }
    if constexpr (RING) {
      if (P.out) {                                                     // one split: this is all there is
        const float f = 1.f / (ll + (P.sink ? exp2f(P.sink[h0 + hh] * 1.4426950408889634f - mm) : 0.f));
        st2(P.out + static_cast<size_t>(b) * P.ld_out + (h0 + hh) * P.vdim + col, make_float2(v.x * f, v.y * f));
        st2(P.out + static_cast<size_t>(b) * P.ld_out + (h0 + hh) * P.vdim + col + 2, make_float2(v.z * f, v.w * f));
        continue;
      }
    }
    const size_t pi = (static_cast<size_t>(b) * P.H + h0 + hh) * P.splits + split;
    *reinterpret_cast<float4*>(P.part_o + pi * vs + col) = v;
    if (col == 0) {
      P.part_ml[2 * pi] = mm * 0.6931471805599453f;
      P.part_ml[2 * pi + 1] = ll;
    }
  }
}

template <int STAGES>
static int gd_smem(int dim, int vdim) {
  const int ring = 16 * gd_pitch(dim) + GD_WARPS * STAGES * GD_KEYS * (gd_pitch(dim) + gd_pitch(vdim));
  const int join = (GD_WARPS * 32 + GD_WARPS * 16 * ((vdim + 7) & ~7)) * 4;
  return ring > join ? ring : join;
}

}  // namespace b200

using namespace b200;

B200_API int b200_gqa_decode_supported(int dim, int vdim) {
  return dim > 0 && vdim > 0 && !(dim & 7) && !(vdim & 7) && dim <= 256 && vdim <= 256;
}

// CTAs of the kernel that fit an SM
B200_API int b200_gqa_decode_per_sm(int dim, int vdim) {
  const int n = 227 * 1024 / (gd_smem<3>(dim, vdim) + 1024);
  return n < 1 ? 1 : n > 4 ? 4 : n;
}

template <bool RING, bool HEADS>
static int gqa_decode_launch(const void* in, const GqaDecode& P, int B, int in_f32, cudaStream_t st) {
  const int chunks = (P.H / P.G + 15) / 16;
  const dim3 grid(P.splits, P.G * chunks, B);
#define GO2(TI, NV, ST)                                                                                                \
  {                                                                                                                    \
    const int smem = gd_smem<ST>(P.dim, P.vdim);                                                                        \
    if (cudaFuncSetAttribute(gqa_decode_kernel<TI, NV, ST, RING, HEADS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3; \
    launch_k(gqa_decode_kernel<TI, NV, ST, RING, HEADS>, grid, dim3(128), smem, st, (const TI*)in, P);                         \
  }
#define GO(TI)                                          \
  {                                                     \
    if (P.vdim <= 64) GO2(TI, 4, 3)                     \
    else if (P.vdim <= 96) GO2(TI, 6, 3)                \
    else if (P.vdim <= 128) GO2(TI, 8, 3)               \
    else GO2(TI, 16, 3)                                 \
  }
  if (in_f32) GO(float) else GO(__nv_bfloat16)
#undef GO
#undef GO2
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

static bool gqa_decode_ok(const GqaDecode& P, int B) {
  return b200_gqa_decode_supported(P.dim, P.vdim) && B > 0 && B <= 65535 && P.H > 0 && P.G > 0 && P.H % P.G == 0 && P.splits >= 1 && P.splits <= 32 &&
         !(P.ld_kv & 7) && !(P.kv_v & 7) && P.cap > 0 && !(reinterpret_cast<uintptr_t>(P.cache) & 15);
}

B200_API int b200_gqa_decode(const void* in, const GqaDecode* Pp, int B, int in_f32, void* stream) {
  if (!gqa_decode_ok(*Pp, B) || Pp->bias_len <= 0) return -1;
  return gqa_decode_launch<false, false>(in, *Pp, B, in_f32, reinterpret_cast<cudaStream_t>(stream));
}

// The RING form; `out` is written with a single split, the partials otherwise.
B200_API int b200_ring_decode(const void* in, const GqaDecode* Pp, int B, int in_f32, void* stream) {
  const GqaDecode& P = *Pp;
  if (!gqa_decode_ok(P, B) || P.size <= 0 || P.rot < 0 || (P.rot & 1) || P.rot > P.dim || (P.rot && (!P.cosT || !P.sinT)) || !P.q_norm != !P.k_norm ||
      (P.lam && !P.first) || P.softcap < 0.f || P.keep < 0 || (P.keep && P.chunked) || (P.head_norm && P.q_norm)) return -1;
  if (((P.ld_in | P.off_k | P.off_v | P.ld_first | P.ld_fout) & 7) ||
      ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(P.q_norm) | reinterpret_cast<uintptr_t>(P.k_norm) | reinterpret_cast<uintptr_t>(P.cosT) |
        reinterpret_cast<uintptr_t>(P.sinT) | reinterpret_cast<uintptr_t>(P.in_bias) | reinterpret_cast<uintptr_t>(P.first) | reinterpret_cast<uintptr_t>(P.first_out)) & 15)) return -1;
  if (P.splits == 1 ? (!P.out || (P.ld_out & 7) || (reinterpret_cast<uintptr_t>(P.out) & 15)) : (P.out || !P.part_o || !P.part_ml)) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return P.keep || P.head_norm || P.in_bias ? gqa_decode_launch<true, true>(in, P, B, in_f32, st) : gqa_decode_launch<true, false>(in, P, B, in_f32, st);
}
