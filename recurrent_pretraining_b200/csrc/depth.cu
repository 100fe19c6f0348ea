// Residual stream of layered decoders that add normed sublayer outputs and average over depth:
//   * depth_norm      : x = x0 + norm(a) on the fp32 stream, RMS norms over equal groups of columns; at the end of a layer x is kept and
//                       replaced by a weighted sum of the embedding output and all layer results so far
//   * group_norm_rows : gathered rows of the final norm
// Storage types: bf16 (serving) or fp32; arithmetic is fp32.  This file is built without fast-math approximations.
#include "rowops.cuh"

namespace b200 {

struct DepthArgs {
  int E, groups, ld_a, ld_h, clear, nzero;
  float eps;
  const float* w;                 // norm weights
  const float* bias;              // on the sublayer output; null: none
  const float* x0;                // stream before (may be x)
  float* x;                       // stream behind
  float* zero;                    // second accumulator, re-armed here
  // sum over depth: x = sum_(j < n_past) dwa[j] past[j] + dwa[n_past] (result), the result kept as past[n_past] with `keep`
  int n_past, keep;               // n_past 0: no sum
  size_t past_pitch;              // elements between the stored results
  float* past;                    // [.., rows, E]
  const float* dwa;
  // sublayer output that is still a sum: see sublayer_cols
  int top, ld_mix, ld_shared;
  const int* slot;
  const float* weight;
  const void *mix_h, *shared;
};

// Root mean squares of the groups from the sums of squares of pieces of `piece` columns: rs[g] = 1 / rms.
template <int THREADS>
__device__ __forceinline__ void group_factors(const float* sq, int per_group, int groups, int cols, float eps, float* rs) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int g = warp; g < groups; g += THREADS / 32) {
    float s = 0.f;
    for (int i = lane; i < per_group; i += 32) s += sq[g * per_group + i];
    s = warp_sum(s);
    if (lane == 0) rs[g] = 1.f / sqrtf(s / static_cast<float>(cols) + eps);
  }
  __syncthreads();
}

// One CTA per row; NV pieces of eight columns per thread held in registers; a group is a whole number of pieces.
template <typename TI, typename T, int NV, bool SUM, int THREADS>
__global__ void __launch_bounds__(THREADS)
depth_vec_kernel(TI* __restrict__ a, T* __restrict__ h, const DepthArgs A) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];                    // [pieces] sums of squares, [groups] factors
  __shared__ float red[THREADS / 32];
  const size_t row = blockIdx.x;
  const int nvec = A.E >> 3, per = nvec / A.groups;
  float* rs = sm + nvec;
  float s[NV][8], xv[NV][8];
  TI* ar = a + row * A.ld_a;
  float total = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = threadIdx.x + k * THREADS;
    if (i < nvec) {
      ld8(A.x0 + row * A.E + 8 * i, xv[k]);
      if constexpr (SUM) sublayer_cols<8, TI, T>(A, a, row, 8 * i, s[k]);
      else ld8(ar + 8 * i, s[k]);
      if (A.clear) clear8(ar + 8 * i);
      if (A.bias) {
        float b[8];
        ld8(A.bias + 8 * i, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) s[k][j] += b[j];
      }
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += s[k][j] * s[k][j];
      if (A.groups > 1) sm[i] = ss;
      total += ss;
    }
  }
  for (int i = threadIdx.x; i < A.nzero; i += THREADS) A.zero[row * A.nzero + i] = 0.f;
  float r1 = 0.f;
  if (A.groups > 1) {
    __syncthreads();
    group_factors<THREADS>(sm, per, A.groups, A.E / A.groups, A.eps, rs);
  } else {
    r1 = 1.f / sqrtf(block_total<THREADS>(total, red) / static_cast<float>(A.E) + A.eps);
  }
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = threadIdx.x + k * THREADS;
    if (i < nvec) {
      const size_t at = row * A.E + 8 * i;
      const float r = A.groups > 1 ? rs[i / per] : r1;
      float wv[8];
      ld8(A.w + 8 * i, wv);
#pragma unroll
      for (int j = 0; j < 8; ++j) xv[k][j] += s[k][j] * r * wv[j];
      if (A.n_past > 0) {
        if (A.keep) st8(A.past + A.n_past * A.past_pitch + at, xv[k]);
        const float own = A.dwa[A.n_past];
#pragma unroll
        for (int j = 0; j < 8; ++j) xv[k][j] *= own;
        int p = 0;
        for (; p + 4 <= A.n_past; p += 4) {        // four results on their way at a time
          float y[4][8];
#pragma unroll
          for (int u = 0; u < 4; ++u) ld8(A.past + (p + u) * A.past_pitch + at, y[u]);
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            const float f = A.dwa[p + u];
#pragma unroll
            for (int j = 0; j < 8; ++j) xv[k][j] += f * y[u][j];
          }
        }
        for (; p < A.n_past; ++p) {
          float y[8];
          ld8(A.past + p * A.past_pitch + at, y);
          const float f = A.dwa[p];
#pragma unroll
          for (int j = 0; j < 8; ++j) xv[k][j] += f * y[j];
        }
      }
      st8(A.x + at, xv[k]);
      st8(h + row * A.ld_h + 8 * i, xv[k]);
    }
  }
}

// Any width: several passes over the row, a warp per group for the norm.
template <typename TI, typename T, bool SUM>
__global__ void __launch_bounds__(256)
depth_kernel(TI* __restrict__ a, T* __restrict__ h, const DepthArgs A) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float rs[];                    // [groups]
  const size_t row = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, per = A.E / A.groups;
  TI* ar = a + row * A.ld_a;
  for (int i = threadIdx.x; i < A.nzero; i += 256) A.zero[row * A.nzero + i] = 0.f;
  auto in = [&](int i) {
    float v;
    if constexpr (SUM) sublayer_cols<1, TI, T>(A, a, row, i, &v);
    else v = ldf(ar + i);
    return v + (A.bias ? A.bias[i] : 0.f);
  };
  for (int g = warp; g < A.groups; g += 8) {
    float ss = 0.f;
    for (int i = lane; i < per; i += 32) {
      const float v = in(g * per + i);
      ss += v * v;
    }
    ss = warp_sum(ss);
    if (lane == 0) rs[g] = 1.f / sqrtf(ss / static_cast<float>(per) + A.eps);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < A.E; i += 256) {
    const size_t at = row * A.E + i;
    float v = A.x0[at] + in(i) * rs[i / per] * A.w[i];
    if (A.clear) stf(ar + i, 0.f);
    if (A.n_past > 0) {
      if (A.keep) A.past[A.n_past * A.past_pitch + at] = v;
      v *= A.dwa[A.n_past];
      for (int p = 0; p < A.n_past; ++p) v += A.dwa[p] * A.past[p * A.past_pitch + at];
    }
    A.x[at] = v;
    stf(h + row * A.ld_h + i, v);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
group_norm_rows_kernel(const float* __restrict__ x, const int* __restrict__ idx, const float* __restrict__ w, T* __restrict__ y, int ld_y,
                       int E, int groups, float eps) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];                    // [256] partial sums, [groups] factors
  const float* xr = x + static_cast<size_t>(idx ? idx[blockIdx.x] : static_cast<int>(blockIdx.x)) * E;
  const int per = E / groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* rs = sm + 8;
  if (groups == 1) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < E; i += 256) ss += xr[i] * xr[i];
    ss = block_total<256>(ss, sm);
    if (threadIdx.x == 0) rs[0] = 1.f / sqrtf(ss / static_cast<float>(E) + eps);
  } else {
    for (int g = warp; g < groups; g += 8) {
      float ss = 0.f;
      for (int i = lane; i < per; i += 32) {
        const float v = xr[g * per + i];
        ss += v * v;
      }
      ss = warp_sum(ss);
      if (lane == 0) rs[g] = 1.f / sqrtf(ss / static_cast<float>(per) + eps);
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < E; i += 256) stf(y + static_cast<size_t>(blockIdx.x) * ld_y + i, xr[i] * rs[i / per] * w[i]);
}

}  // namespace b200

using namespace b200;
typedef __nv_bfloat16 bf16_t;
#define STREAM reinterpret_cast<cudaStream_t>(stream)
#define DONE (cudaGetLastError() == cudaSuccess ? 0 : -2)

template <typename TI, typename T, bool SUM>
static int launch_depth(void* a, void* h, const DepthArgs& A, int rows, cudaStream_t st) {
  const uintptr_t addr = reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(A.x0) | reinterpret_cast<uintptr_t>(A.x) |
                         reinterpret_cast<uintptr_t>(A.w) | reinterpret_cast<uintptr_t>(A.bias) | reinterpret_cast<uintptr_t>(A.past) |
                         reinterpret_cast<uintptr_t>(A.mix_h) | reinterpret_cast<uintptr_t>(A.shared);
  const bool vec = !(addr & 15) && !((A.E | (A.E / A.groups) | A.ld_a | A.ld_h | A.ld_mix | A.ld_shared) & 7) && !(A.past_pitch & 3);
  const int nvec = A.E / 8;
  const size_t smem = (vec ? nvec + A.groups : A.groups) * sizeof(float);
  if (smem > 48 * 1024) return -1;
#define GO(NV, TH) launch_k(depth_vec_kernel<TI, T, NV, SUM, TH>, dim3(rows), dim3(TH), smem, st, (TI*)a, (T*)h, A)
  if (vec && nvec <= 128) GO(1, 128);
  else if (vec && nvec <= 256) GO(1, 256);
  else if (vec && nvec <= 512) GO(2, 256);
  else if (vec && nvec <= 1024) GO(4, 256);
  else launch_k(depth_kernel<TI, T, SUM>, dim3(rows), dim3(256), A.groups * sizeof(float), st, (TI*)a, (T*)h, A);
#undef GO
  return DONE;
}

// a: sublayer output (fp32 with in_f32), h: operand copy of the new stream.
B200_API int b200_depth_norm(void* a, void* h, const DepthArgs* Ap, int rows, int in_f32, int f32, void* stream) {
  const DepthArgs A = *Ap;
  if (rows <= 0 || A.E <= 0 || A.groups <= 0 || A.E % A.groups || !a || !h || !A.x0 || !A.x || !A.w || (A.clear && !in_f32) || (f32 && !in_f32) ||
      (A.nzero && !A.zero) || (A.n_past && (!A.past || !A.dwa)) || A.n_past < 0) return -1;
  if (A.top && (!in_f32 || A.top < 0 || A.clear || !A.slot || !A.weight || !A.mix_h)) return -1;
  if (A.top) return f32 ? launch_depth<float, float, true>(a, h, A, rows, STREAM) : launch_depth<float, bf16_t, true>(a, h, A, rows, STREAM);
  if (f32) return launch_depth<float, float, false>(a, h, A, rows, STREAM);
  if (in_f32) return launch_depth<float, bf16_t, false>(a, h, A, rows, STREAM);
  return launch_depth<bf16_t, bf16_t, false>(a, h, A, rows, STREAM);
}

B200_API int b200_group_norm_rows(const float* x, const int* idx, const float* w, void* y, int ld_y, int rows, int E, int groups, float eps,
                                  int f32, void* stream) {
  if (rows <= 0) return 0;
  const size_t smem = (8 + groups) * sizeof(float);
  if (E <= 0 || groups <= 0 || E % groups || smem > 48 * 1024) return -1;
  if (f32) launch_k(group_norm_rows_kernel<float>, dim3(rows), dim3(256), smem, STREAM, x, idx, w, (float*)y, ld_y, E, groups, eps);
  else launch_k(group_norm_rows_kernel<bf16_t>, dim3(rows), dim3(256), smem, STREAM, x, idx, w, (bf16_t*)y, ld_y, E, groups, eps);
  return DONE;
}
