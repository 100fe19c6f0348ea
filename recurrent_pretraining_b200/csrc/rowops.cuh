// Row helpers of the layered decoders' kernels: typed element access (bf16 or fp32 storage, fp32 arithmetic), block sums.
#pragma once
#include "common.cuh"

namespace b200 {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ void stf(T* p, float v);
template <> __device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stf<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// two neighbouring elements (address aligned to the pair)
template <typename T> __device__ __forceinline__ float2 ld2(const T* p);
template <> __device__ __forceinline__ float2 ld2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 ld2<__nv_bfloat16>(const __nv_bfloat16* p) {
  return unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p));
}
__device__ __forceinline__ void st2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void st2(__nv_bfloat16* p, float2 v) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(v.x, v.y); }
// four neighbouring elements
__device__ __forceinline__ void ld4(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void ld4(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 q = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(q.x), b = unpack_bf16x2(q.y);
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
// eight neighbouring elements (16-byte aligned rows)
__device__ __forceinline__ void ld8(const float* p, float (&v)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void ld8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 q = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = unpack_bf16x2(w[j]);
    v[2 * j] = f.x;
    v[2 * j + 1] = f.y;
  }
}
__device__ __forceinline__ void st8(float* p, const float (&v)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void st8(__nv_bfloat16* p, const float (&v)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]),
                                            pack_bf16x2(v[6], v[7]));
}
__device__ __forceinline__ void clear8(float* p) {
  reinterpret_cast<float4*>(p)[0] = make_float4(0.f, 0.f, 0.f, 0.f);
  reinterpret_cast<float4*>(p)[1] = make_float4(0.f, 0.f, 0.f, 0.f);
}
__device__ __forceinline__ void clear8(__nv_bfloat16*) {}

template <int THREADS>
__device__ __forceinline__ float block_total(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();   // the previous use of `red` is over
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) t += red[i];
  return t;
}
__device__ __forceinline__ float sigmoid_f(float v) { return 1.f / (1.f + expf(-v)); }
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }
// factor on the queries of position p
__device__ __forceinline__ float query_temperature(int p, int every, float coef) {
  return 1.f + coef * logf(static_cast<float>((p + 1) / every + 1));
}
// slot of position p in a ring of `cap` slots whose first `keep` hold the sequence's first positions for good
__device__ __forceinline__ int ring_slot(int p, int cap, int keep) { return p < cap ? p : keep + (p - keep) % (cap - keep); }
// log(1 + exp(v))
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float silu_f(float v) { return v / (1.f + expf(-v)); }

// Eight columns (V = 8) or one of the output of a sublayer that is still a sum (`Args`: SandwichArgs or DepthArgs): row `row` is
// sum_k weight[row, k] a[slot[row, k]], with mix_h[row] in place of a row whose slot is negative, + weight[row, top] shared[row].
template <int V, typename TI, typename T, typename Args>
__device__ __forceinline__ void sublayer_cols(const Args& A, const TI* a, size_t row, int i, float* v) {
  auto load = [](const auto* p, float* o) {
    if constexpr (V == 8) ld8(p, *reinterpret_cast<float(*)[8]>(o));
    else *o = ldf(p);
  };
  const int* sl = A.slot + row * A.top;
  const float* wt = A.weight + row * (A.top + 1);
#pragma unroll
  for (int j = 0; j < V; ++j) v[j] = 0.f;
  for (int k0 = 0; k0 < A.top; k0 += 4) {                 // four rows on their way at a time
    float y[4][V], f[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      f[u] = 0.f;
      if (k0 + u < A.top) {
        const int s = sl[k0 + u];
        f[u] = wt[k0 + u];
        if (s < 0) load(reinterpret_cast<const T*>(A.mix_h) + row * A.ld_mix + i, y[u]);
        else load(a + static_cast<size_t>(s) * A.ld_a + i, y[u]);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) y[u][j] = 0.f;
      }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u)
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] += f[u] * y[u][j];
  }
  if (A.shared) {
    float y[V];
    load(reinterpret_cast<const TI*>(A.shared) + row * A.ld_shared + i, y);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] += wt[A.top] * y[j];
  }
}

}  // namespace b200
