// Mixture-of-experts feed-forward around the grouped matrix products:
//   * moe_router_logits : product of a decode step's rows with the router, fp32 operands
//   * moe_route         : softmax or sigmoid of the router outputs, choice of the best ones (scores plus correction; of the best groups
//                         only), weights (normalised or not), rank of every choice inside its expert
//   * moe_plan          : first slot of every expert (rows padded to whole tiles), expert of every tile
//   * moe_dispatch      : rows into their experts' slots
//   * moe_route_rows    : the three in one CTA for the few rows of a decode step, slots without padding
//   * moe_rows          : product of a decode step's rows with their experts' weights: a stream of weights through mma.sync,
//                         fragments straight from memory
//   * moe_combine       : weighted sum of a token's experts, identity experts and the gated shared expert (prompts; in a decode step
//                         the norm that reads the sum forms it: sandwich_norm in memory.cu)
// Storage types: bf16 (serving) or fp32; arithmetic is fp32.  This file is built without fast-math approximations.
#include "rowops.cuh"

namespace b200 {

constexpr int MOE_MAX_OUT = 1024;       // router outputs

struct RouteArgs {
  int experts, outputs, top;            // outputs: experts and identity experts
  int ld_z, gate;                       // gate: column `outputs` of z is the shared expert's gate
  int sigmoid, normalize;               // scores are sigmoids (else a softmax); the chosen ones are divided by their sum
  int groups, keep;                     // equal groups of neighbouring outputs; only those of the best `keep` groups can be chosen
  const float* correction;              // [outputs]; null: none
  int* idx;                             // [T, top] chosen outputs
  float* weight;                        // [T, top + 1] their weights; then the gate's sigmoid
};

// Best of the lanes' (value, index) pairs; the lower index among equals.
__device__ __forceinline__ void warp_best(float& best, int& at) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ob = __shfl_xor_sync(0xffffffffu, best, o);
    const int oa = __shfl_xor_sync(0xffffffffu, at, o);
    if (ob > best || (ob == best && oa < at)) { best = ob; at = oa; }
  }
}

// Scores and choice for one token by one warp; s, c: [outputs] scratch of the warp in shared memory.
__device__ __forceinline__ void route_token(const RouteArgs& R, const float* z, size_t t, float* s, float* c) {
  const int lane = threadIdx.x & 31;
  float sum = 1.f;
  if (R.sigmoid) {
    for (int i = lane; i < R.outputs; i += 32) s[i] = sigmoid_f(z[i]);
  } else {
    float m = -INFINITY;
    for (int i = lane; i < R.outputs; i += 32) m = fmaxf(m, z[i]);
    m = warp_max(m);
    sum = 0.f;
    for (int i = lane; i < R.outputs; i += 32) {
      const float e = expf(z[i] - m);
      s[i] = e;
      sum += e;
    }
    sum = warp_sum(sum);
  }
  for (int i = lane; i < R.outputs; i += 32) {
    s[i] = s[i] / sum;
    c[i] = s[i] + (R.correction ? R.correction[i] : 0.f);
  }
  __syncwarp();
  if (R.keep < R.groups) {                // c keeps the scores of the best groups only; a lane owns every 32nd group
    const int per = R.outputs / R.groups;
    auto strength = [&](int g) {
      float a = -INFINITY, b = -INFINITY;                 // the two largest
      for (int i = g * per; i < (g + 1) * per; ++i) {
        const float v = c[i];
        if (v > a) { b = a; a = v; }
        else if (v > b) b = v;
      }
      return per > 1 ? a + b : a;
    };
    float last = INFINITY;                // strength and index of the group chosen before
    int last_at = -1;
    for (int k = 0; k < R.keep; ++k) {
      float best = -INFINITY;
      int at = R.groups;
      for (int g = lane; g < R.groups; g += 32) {
        const float v = strength(g);
        if ((v < last || (v == last && g > last_at)) && (v > best || (v == best && g < at))) { best = v; at = g; }
      }
      warp_best(best, at);
      last = best;
      last_at = at;
    }
    // the groups behind the last chosen one, in order of strength, are out
    for (int g = lane; g < R.groups; g += 32) {
      const float v = strength(g);
      if (v < last || (v == last && g > last_at))
        for (int i = g * per; i < (g + 1) * per; ++i) c[i] = -INFINITY;
    }
    __syncwarp();
  }
  float total = 0.f, mine = 0.f;
  for (int k = 0; k < R.top; ++k) {
    float best = -INFINITY;
    int at = R.outputs;
    for (int i = lane; i < R.outputs; i += 32)
      if (c[i] > best) { best = c[i]; at = i; }
    warp_best(best, at);
    at = min(at, R.outputs - 1);        // only if every score left is NaN
    const float w = s[at];
    total += w;
    __syncwarp();
    if (lane == 0) {
      c[at] = -INFINITY;
      R.idx[t * R.top + k] = at;
    }
    if ((k & 31) == lane) mine = w;
    if ((k & 31) == 31 || k + 1 == R.top) {               // up to 32 weights at a time, normalised below
      const int k0 = k & ~31;
      if (k0 + lane <= k) R.weight[t * (R.top + 1) + k0 + lane] = mine;
    }
    __syncwarp();
  }
  if (R.normalize)
    for (int k = lane; k < R.top; k += 32) R.weight[t * (R.top + 1) + k] /= total + 1e-20f;
  if (lane == 0) R.weight[t * (R.top + 1) + R.top] = R.gate ? sigmoid_f(z[R.outputs]) : 0.f;
}

// z[b, r] = x[b] . w[r]: CTA per router output (fp32 operands; bf16 ones go through moe_rows)
template <typename T>
__global__ void __launch_bounds__(128)
moe_router_logits_kernel(const T* __restrict__ x, int ld_x, const T* __restrict__ w, int ld_w, float* __restrict__ z, int ld_z, int B, int E) {
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* wr = w + static_cast<size_t>(r) * ld_w;
  for (int b = warp; b < B; b += 4) {
    const T* xr = x + static_cast<size_t>(b) * ld_x;
    float s = 0.f;
    int i = 8 * lane;
#pragma unroll 4
    for (; i + 8 <= E; i += 256) {
      float a[8], c[8];
      ld8(xr + i, a);
      ld8(wr + i, c);
#pragma unroll
      for (int j = 0; j < 8; ++j) s += a[j] * c[j];
    }
    for (; i < E; ++i) s += ldf(xr + i) * ldf(wr + i);    // the last lane with columns left
    s = warp_sum(s);
    if (lane == 0) z[static_cast<size_t>(b) * ld_z + r] = s;
  }
}

// Eight warps, `per` tokens: choices are ranked inside their expert first within the CTA, then across CTAs.
__global__ void __launch_bounds__(256)
moe_route_kernel(const float* __restrict__ z, const RouteArgs R, int* __restrict__ count, int* __restrict__ rank, int T, int per) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5;
  int* hist = reinterpret_cast<int*>(sm + 16 * R.outputs);       // [experts]: choices of this CTA, then their first rank
  for (int i = threadIdx.x; i < R.experts; i += 256) hist[i] = 0;
  const int t0 = blockIdx.x * per, n = min(per, T - t0);
  for (int j = warp; j < n; j += 8)
    route_token(R, z + static_cast<size_t>(t0 + j) * R.ld_z, t0 + j, sm + 2 * warp * R.outputs, sm + (2 * warp + 1) * R.outputs);
  __syncthreads();
  for (int i = threadIdx.x; i < n * R.top; i += 256) {
    const int e = R.idx[static_cast<size_t>(t0) * R.top + i];
    if (e < R.experts) rank[static_cast<size_t>(t0) * R.top + i] = atomicAdd(&hist[e], 1);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < R.experts; i += 256) hist[i] = hist[i] ? atomicAdd(&count[i], hist[i]) : 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n * R.top; i += 256) {
    const int e = R.idx[static_cast<size_t>(t0) * R.top + i];
    if (e < R.experts) rank[static_cast<size_t>(t0) * R.top + i] += hist[e];
  }
}

// One CTA.  offset[e]: first slot of expert e, padded to `rows` slots; tile_expert[i]: expert of slots [i rows, (i + 1) rows);
// n_tiles: their number.
__global__ void __launch_bounds__(256)
moe_plan_kernel(const int* __restrict__ count, int experts, int rows, int* __restrict__ offset, int* __restrict__ tile_expert,
                int* __restrict__ n_tiles) {
  __shared__ int part[256];
  const int per = (experts + 255) / 256, e0 = min(experts, static_cast<int>(threadIdx.x) * per), e1 = min(experts, e0 + per);
  int tiles = 0;
  for (int e = e0; e < e1; ++e) tiles += (count[e] + rows - 1) / rows;
  part[threadIdx.x] = tiles;
  __syncthreads();
  for (int o = 1; o < 256; o <<= 1) {
    const int v = static_cast<int>(threadIdx.x) >= o ? part[threadIdx.x - o] : 0;
    __syncthreads();
    part[threadIdx.x] += v;
    __syncthreads();
  }
  int at = part[threadIdx.x] - tiles;
  for (int e = e0; e < e1; ++e) {
    offset[e] = at * rows;
    const int n = (count[e] + rows - 1) / rows;
    for (int i = 0; i < n; ++i) tile_expert[at++] = e;
  }
  if (threadIdx.x == 255) *n_tiles = part[255];
}

// CTA per token: its row to the slots of its experts; slot[t, k] = -1 for an identity expert.
__global__ void __launch_bounds__(128)
moe_dispatch_kernel(const uint4* __restrict__ h, int vec_h, uint4* __restrict__ xs, int vec_x, int vec, const int* __restrict__ idx,
                    const int* __restrict__ rank, const int* __restrict__ offset, int* __restrict__ slot, int experts, int top) {
  const size_t t = blockIdx.x;
  const uint4* src = h + t * vec_h;
  for (int i = threadIdx.x; i < top; i += 128) {
    const int e = idx[t * top + i];
    slot[t * top + i] = e < experts ? offset[e] + rank[t * top + i] : -1;
  }
  for (int i = threadIdx.x; i < vec; i += 128) {
    const uint4 v = src[i];
    for (int k = 0; k < top; ++k) {
      const int e = idx[t * top + k];
      if (e < experts) xs[static_cast<size_t>(offset[e] + rank[t * top + k]) * vec_x + i] = v;
    }
  }
}

// A decode step's routing in one CTA: choices and weights, then the slots [first[i], first[i + 1]) of the i-th expert that was
// chosen (active[i]), row[slot], slot[b, k]; n_active: chosen experts.
struct RouteRows {
  int *slot, *active, *first, *row, *n_active;
};
__global__ void __launch_bounds__(1024)
moe_route_rows_kernel(const float* __restrict__ z, const RouteArgs R, const RouteRows A, int B) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];
  const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int* count = reinterpret_cast<int*>(sm + 2 * warps * R.outputs);       // [experts]
  int* base = count + R.experts;                                         // [experts]
  for (int i = threadIdx.x; i < R.experts; i += blockDim.x) count[i] = 0;
  for (int b = warp; b < B; b += warps)
    route_token(R, z + static_cast<size_t>(b) * R.ld_z, b, sm + 2 * warp * R.outputs, sm + (2 * warp + 1) * R.outputs);
  __syncthreads();
  for (int i = threadIdx.x; i < B * R.top; i += blockDim.x) {
    const int e = R.idx[i];
    A.slot[i] = e < R.experts ? atomicAdd(&count[e], 1) : -1;            // rank inside the expert for now
  }
  __syncthreads();
  if (warp == 0) {                                                       // prefix sums over the chosen experts
    int slots = 0, act = 0;
    for (int e0 = 0; e0 < R.experts; e0 += 32) {
      const int e = e0 + lane, n = e < R.experts ? count[e] : 0;
      int inc = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, inc, o);
        if (lane >= o) inc += v;
      }
      const uint32_t some = __ballot_sync(0xffffffffu, n > 0);
      if (n > 0) {
        const int i = act + __popc(some & ((1u << lane) - 1));
        A.active[i] = e;
        A.first[i] = slots + inc - n;
      }
      if (e < R.experts) base[e] = slots + inc - n;
      slots += __shfl_sync(0xffffffffu, inc, 31);
      act += __popc(some);
    }
    if (lane == 0) {
      A.first[act] = slots;
      *A.n_active = act;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < B * R.top; i += blockDim.x) {
    const int e = R.idx[i];
    if (e >= R.experts) continue;
    const int s = base[e] + A.slot[i];
    A.slot[i] = s;
    A.row[s] = i / R.top;
  }
}

// ------------------------------------------------------------------------------------------------ decode products
struct ExpertRows {
  int N, K, ld_w;                       // weights [groups * N, ld_w] bf16, rows padded to eight
  int Ns, Ks, ld_ws;                    // the shared expert's (Ns = 0: none)
  int ld_x, ld_y, ld_xs, ld_ys;         // input and output row pitches (shared: the same or other buffers)
  int B, act;                           // act: 0 none, 1 relu^2, 2 silu gate: an expert's weights are 2 N rows [gate; up]
  const __nv_bfloat16 *w, *ws;
  const __nv_bfloat16 *x, *xs;          // input rows; x is indexed by row[slot] (gather) or by the slot, xs by the token
  int gather;
  void *y, *ys;                         // [slots, ld_y], [B, ld_ys]
  const int *active, *first, *row, *n_active;
};

__device__ __forceinline__ void mma_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// keep the first n of eight bf16 values
__device__ __forceinline__ uint4 keep8(uint4 v, int n) {
  uint32_t* w = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
  for (int i = 0; i < 4; ++i) w[i] = 2 * i + 1 < n ? w[i] : 2 * i < n ? (w[i] & 0xffffu) : 0u;
  return v;
}

__device__ __forceinline__ void cp_async16_zfill(uint32_t dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(on ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// CTA: (16 RG weight rows, chosen expert): RG groups of 16 rows x KW ranges of K, one warp each.  The order of the terms of a dot
// product is free, so a lane takes eight neighbouring columns of its weight rows and of its token as they lie in memory: they
// serve two MMAs.  Weights and tokens pass through a queue in shared memory, several steps of 32 columns in flight: the weights' part
// belongs to the thread alone, and so does the tokens' when the warps stand at different columns (KW > 1: no barriers).  With KW = 1 all
// warps share one copy of the tokens and meet once a step.  NT: groups of eight tokens.  GATED: the sixteen
// rows of a warp are eight gate rows and the eight up rows that belong to them, so that a thread holds both.
template <int NT, int KW>
struct RowsQueue {
  static constexpr bool SHARED_X = KW == 1;
  static constexpr int X_BYTES = SHARED_X ? NT * 512 : NT * 4096, STEP = 8192 + X_BYTES;
  static constexpr int DEPTH = SHARED_X ? 8 : (NT >= 8 ? 5 : 8);
  static constexpr int BYTES = DEPTH * STEP;
};
template <typename TO, int NT, int RG, int KW, bool GATED>
__global__ void __launch_bounds__(256, NT * KW >= 32 ? 1 : 2)
moe_rows_kernel(const ExpertRows P) {
  static_assert(RG * KW == 8, "eight warps");
  using Q = RowsQueue<NT, KW>;
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rg = warp % RG, kw = warp / RG;
  pdl_wait();
  const int shared = P.Ns > 0 ? 1 : 0;
  const bool mine = shared && blockIdx.y == 0;                // the shared expert, which has the most rows, goes first
  int e = 0, s0 = 0, n = P.B;
  if (!mine) {
    const int y = blockIdx.y - shared;
    if (y >= *P.n_active) return;
    e = P.active[y];
    s0 = P.first[y];
    n = P.first[y + 1] - s0;
  }
  const int N = mine ? P.Ns : P.N, K = mine ? P.Ks : P.K, r0 = blockIdx.x * (GATED ? 8 : 16) * RG;
  if (r0 >= N) return;
  const int ldw = mine ? P.ld_ws : P.ld_w, ldx = mine ? P.ld_xs : P.ld_x;
  const __nv_bfloat16* w = mine ? P.ws : P.w + static_cast<size_t>(e) * (GATED ? 2 : 1) * P.N * P.ld_w;
  const __nv_bfloat16* x = mine ? P.xs : P.x;
  const int q = lane & 3, rr = r0 + rg * (GATED ? 8 : 16) + (lane >> 2), r1 = GATED ? N + rr : rr + 8;
  const bool live0 = rr < N, live1 = GATED ? live0 : r1 < N;
  const __nv_bfloat16* w0 = w + static_cast<size_t>(live0 ? rr : 0) * ldw + 8 * q;
  const __nv_bfloat16* w1 = w + static_cast<size_t>(live1 ? r1 : 0) * ldw + 8 * q;
  // this thread's source of token pieces: its own token of every group, or with SHARED_X one piece of one token
  const __nv_bfloat16* xp[Q::SHARED_X ? 1 : NT];
  bool xl[Q::SHARED_X ? 1 : NT];
#pragma unroll
  for (int j = 0; j < (Q::SHARED_X ? 1 : NT); ++j) {
    const int tk = Q::SHARED_X ? threadIdx.x >> 2 : 8 * j + (lane >> 2);
    xl[j] = tk < n && tk < 8 * NT;
    const int s = s0 + (xl[j] ? tk : 0);
    xp[j] = x + static_cast<size_t>(mine ? (xl[j] ? tk : 0) : P.gather ? P.row[s] : s) * ldx + 8 * q;
  }
  const int steps = (K + 31) >> 5, k0 = steps * kw / KW, k1 = steps * (kw + 1) / KW;
  float c[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) c[j][0] = c[j][1] = c[j][2] = c[j][3] = 0.f;
  const uint32_t queue = smem_u32(smem);
  auto request = [&](int k, int slot) {
    const uint32_t d = queue + slot * Q::STEP + threadIdx.x * 16;      // [weights of rows r, of rows r + 8, tokens]
    const bool in = k < k1 && k * 32 + 8 * q < K;
    const int col = in ? k * 32 : 0;
    cp_async16_zfill(d, w0 + col, in && live0);
    cp_async16_zfill(d + 4096, w1 + col, in && live1);
    if constexpr (Q::SHARED_X) {
      if (threadIdx.x < 32 * NT) cp_async16_zfill(d + 8192, xp[0] + col, in && xl[0]);
    } else {
#pragma unroll
      for (int j = 0; j < NT; ++j)
        if (8 * j < n) cp_async16_zfill(d + 8192 + j * 4096, xp[j] + col, in && xl[j]);
    }
  };
  int slot = 0, next = Q::DEPTH - 1;
#pragma unroll
  for (int s = 0; s < Q::DEPTH - 1; ++s) {
    request(k0 + s, s);
    cp_commit();
  }
  for (int k = k0; k < k1; ++k) {
    cp_wait<Q::DEPTH - 2>();
    if constexpr (Q::SHARED_X) __syncthreads();               // the step's tokens are there, and everyone is done with the one before
    request(k + Q::DEPTH - 1, next);
    cp_commit();
    const uint8_t* d = smem + slot * Q::STEP;
    const uint4 a = *reinterpret_cast<const uint4*>(d + threadIdx.x * 16), b = *reinterpret_cast<const uint4*>(d + 4096 + threadIdx.x * 16);
    const uint8_t* dx = d + 8192 + (Q::SHARED_X ? lane : static_cast<int>(threadIdx.x)) * 16;
    const int left = K - (k * 32 + 8 * q);
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      if (8 * j >= n) break;                                  // uniform over the CTA
      uint4 v = *reinterpret_cast<const uint4*>(dx + j * (Q::SHARED_X ? 512 : 4096));
      if (left > 0 && left < 8) v = keep8(v, left);           // padding columns of a row are not initialised
      mma_16816(c[j], a.x, b.x, a.y, b.y, v.x, v.y);
      mma_16816(c[j], a.z, b.z, a.w, b.w, v.z, v.w);
    }
    slot = slot + 1 == Q::DEPTH ? 0 : slot + 1;
    next = next + 1 == Q::DEPTH ? 0 : next + 1;
  }
  cp_wait<0>();
  // c[j][0..1]: row rr, tokens 8 j + 2 q + {0, 1}; c[j][2..3]: row rr + 8
  float* part = reinterpret_cast<float*>(smem);               // [KW - 1][RG][16][8 NT + 1], over the queue
  constexpr int LP = 8 * NT + 1;
  if constexpr (KW > 1) {
    __syncthreads();
    if (kw) {
      float* pp = part + ((kw - 1) * RG + rg) * 16 * LP;
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) pp[((lane >> 2) + 8 * (i >> 1)) * LP + 8 * j + 2 * q + (i & 1)] = c[j][i];
    }
    __syncthreads();
    if (kw) return;
  }
  TO* y = reinterpret_cast<TO*>(mine ? P.ys : P.y) + (mine ? 0 : static_cast<size_t>(s0) * P.ld_y);
  const int ldy = mine ? P.ld_ys : P.ld_y;
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    if (8 * j >= n) break;
    float v[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (lane >> 2) + 8 * (i >> 1), tk = 8 * j + 2 * q + (i & 1);
      v[i] = c[j][i];
#pragma unroll
      for (int g = 0; g < KW - 1; ++g) v[i] += part[(g * RG + rg) * 16 * LP + r * LP + tk];
    }
    if constexpr (GATED) {
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int tk = 8 * j + 2 * q + i;
        if (tk < n && live0) stf(y + static_cast<size_t>(tk) * ldy + rr, silu_f(v[i]) * v[i + 2]);
      }
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = (lane >> 2) + 8 * (i >> 1), tk = 8 * j + 2 * q + (i & 1);
        if (P.act == 1) {
          v[i] = fmaxf(v[i], 0.f);
          v[i] *= v[i];
        }
        if (tk < n && r0 + rg * 16 + r < N) stf(y + static_cast<size_t>(tk) * ldy + r0 + rg * 16 + r, v[i]);
      }
    }
  }
}

template <typename TO, int NT, int RG, int KW, bool GATED = false>
static int launch_rows(const ExpertRows& P, int max_active, cudaStream_t st) {
  constexpr int QUEUE = RowsQueue<NT, KW>::BYTES, PART = (KW - 1) * RG * 16 * (8 * NT + 1) * 4, SMEM = QUEUE > PART ? QUEUE : PART;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(moe_rows_kernel<TO, NT, RG, KW, GATED>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM) != cudaSuccess) return -3;
    configured = true;
  }
  const int rows = P.N > P.Ns ? P.N : P.Ns;
  constexpr int OUT = (GATED ? 8 : 16) * RG;         // results per CTA and token
  const dim3 grid((rows + OUT - 1) / OUT, max_active + (P.Ns ? 1 : 0));
  launch_k(moe_rows_kernel<TO, NT, RG, KW, GATED>, grid, dim3(256), static_cast<size_t>(SMEM), st, P);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// ------------------------------------------------------------------------------------------------ sum of the experts
// out[t] = sum_k weight[t, k] * (slot[t, k] < 0 ? h[t] : y[slot[t, k]]) + weight[t, top] * ys[t]
template <typename T, int W>
__global__ void __launch_bounds__(256)
moe_combine_kernel(const T* __restrict__ h, int ld_h, const T* __restrict__ y, int ld_y, const T* __restrict__ ys, int ld_ys,
                   const int* __restrict__ slot, const float* __restrict__ weight, T* __restrict__ out, int ld_out, int E, int top) {
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int* sl = slot + t * top;
  const float* wt = weight + t * (top + 1);
  for (int i = threadIdx.x * W; i < E; i += 256 * W) {
    float acc[W], v[W];
#pragma unroll
    for (int j = 0; j < W; ++j) acc[j] = 0.f;
    for (int k = 0; k < top; ++k) {
      const int s = sl[k];
      const float f = wt[k];
      if constexpr (W == 8) {
        if (s < 0) ld8(h + t * ld_h + i, v);
        else ld8(y + static_cast<size_t>(s) * ld_y + i, v);
      } else {
        v[0] = s < 0 ? ldf(h + t * ld_h + i) : ldf(y + static_cast<size_t>(s) * ld_y + i);
      }
#pragma unroll
      for (int j = 0; j < W; ++j) acc[j] += f * v[j];
    }
    if (ys) {
      const float f = wt[top];
      if constexpr (W == 8) ld8(ys + t * ld_ys + i, v);
      else v[0] = ldf(ys + t * ld_ys + i);
#pragma unroll
      for (int j = 0; j < W; ++j) acc[j] += f * v[j];
    }
    if constexpr (W == 8) st8(out + t * ld_out + i, acc);
    else stf(out + t * ld_out + i, acc[0]);
  }
}

}  // namespace b200

using namespace b200;
typedef __nv_bfloat16 bf16_t;
#define STREAM reinterpret_cast<cudaStream_t>(stream)
#define DONE (cudaGetLastError() == cudaSuccess ? 0 : -2)

B200_API int b200_moe_max_outputs() { return MOE_MAX_OUT; }

B200_API int b200_moe_router_logits(const void* x, int ld_x, const void* w, int ld_w, float* z, int ld_z, int B, int R, int E, int f32,
                                    void* stream) {
  if (B <= 0 || R <= 0 || E <= 0 || ld_z < R || !f32 || ((ld_x | ld_w) & 7) || ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w)) & 15)) return -1;
  launch_k(moe_router_logits_kernel<float>, dim3(R), dim3(128), 0, STREAM, (const float*)x, ld_x, (const float*)w, ld_w, z, ld_z, B, E);
  return DONE;
}

static bool route_ok(const RouteArgs& R) {
  return R.experts > 0 && R.outputs >= R.experts && R.outputs <= MOE_MAX_OUT && R.top > 0 && R.top <= R.outputs && R.ld_z >= R.outputs + (R.gate ? 1 : 0) &&
         R.groups > 0 && R.outputs % R.groups == 0 && R.keep > 0 && R.keep <= R.groups && R.top <= R.outputs / R.groups * R.keep && R.idx && R.weight;
}

// z: [T, ld_z] router logits; count: [experts], zero on entry; rank: [T, top]; tile_expert: [max_tiles], rows slots each.
B200_API int b200_moe_route(const float* z, const RouteArgs* Rp, int* count, int* rank, int T, void* stream) {
  const RouteArgs R = *Rp;
  if (T <= 0 || !route_ok(R)) return -1;
  const int smem = (16 * R.outputs + R.experts) * 4;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
  const int per = T <= 16384 ? 8 : 32;      // few tokens per CTA: short; many: fewer additions to the counts
  moe_route_kernel<<<(T + per - 1) / per, 256, smem, STREAM>>>(z, R, count, rank, T, per);
  return DONE;
}

B200_API int b200_moe_plan(const int* count, int experts, int rows, int* offset, int* tile_expert, int* n_tiles, void* stream) {
  if (experts <= 0 || rows <= 0) return -1;
  moe_plan_kernel<<<1, 256, 0, STREAM>>>(count, experts, rows, offset, tile_expert, n_tiles);
  return DONE;
}

// rows of `row_bytes` (a multiple of 16), pitches in bytes
B200_API int b200_moe_dispatch(const void* h, int pitch_h, void* xs, int pitch_x, int row_bytes, const int* idx, const int* rank, const int* offset,
                               int* slot, int experts, int top, int T, void* stream) {
  if (T <= 0 || ((pitch_h | pitch_x | row_bytes) & 15) || row_bytes > pitch_h || row_bytes > pitch_x) return -1;
  moe_dispatch_kernel<<<T, 128, 0, STREAM>>>((const uint4*)h, pitch_h / 16, (uint4*)xs, pitch_x / 16, row_bytes / 16, idx, rank, offset, slot, experts, top);
  return DONE;
}

B200_API int b200_moe_route_rows(const float* z, const RouteArgs* Rp, const RouteRows* Ap, int B, void* stream) {
  const RouteArgs R = *Rp;
  if (B <= 0 || B > 64 || !route_ok(R)) return -1;
  int warps = B < 32 ? B : 32;
  while (warps > 1 && (2 * warps * R.outputs + 2 * R.experts) * 4 > 200 * 1024) warps /= 2;
  const int smem = (2 * warps * R.outputs + 2 * R.experts) * 4;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(moe_route_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
  launch_k(moe_route_rows_kernel, dim3(1), dim3(32 * warps), static_cast<size_t>(smem), STREAM, z, R, *Ap, B);
  return DONE;
}

// max_active: most experts that can have been chosen (0: only the shared expert's matrix).  narrow: matrices of few rows.
B200_API int b200_moe_rows(const ExpertRows* Pp, int max_active, int out_f32, int narrow, void* stream) {
  const ExpertRows P = *Pp;
  if (P.B <= 0 || P.B > 64 || max_active < 0 || max_active > 65534 || P.N < 0 || P.Ns < 0 || (!P.Ns && !max_active)) return -1;
  if ((max_active && (P.N <= 0 || P.K <= 0 || !P.w || !P.x || !P.y || !P.active || !P.first || !P.n_active || (P.gather && !P.row))) ||
      (P.Ns && (P.Ks <= 0 || !P.ws || !P.xs || !P.ys))) return -1;
  if (((P.ld_w | P.ld_x | P.ld_ws | P.ld_xs) & 7) || ((reinterpret_cast<uintptr_t>(P.w) | reinterpret_cast<uintptr_t>(P.ws) | reinterpret_cast<uintptr_t>(P.x) |
                                                      reinterpret_cast<uintptr_t>(P.xs)) & 15)) return -1;
  if (P.act < 0 || P.act > 2) return -1;
  if (P.act == 2) {
    if (P.Ns || out_f32 || narrow) return -1;
    if (P.B <= 2) return launch_rows<bf16_t, 1, 1, 8, true>(P, max_active, STREAM);
    if (P.B <= 8) return launch_rows<bf16_t, 1, 2, 4, true>(P, max_active, STREAM);
    if (P.B <= 16) return launch_rows<bf16_t, 2, 4, 2, true>(P, max_active, STREAM);
    if (P.B <= 32) return launch_rows<bf16_t, 4, 8, 1, true>(P, max_active, STREAM);
    return launch_rows<bf16_t, 8, 8, 1, true>(P, max_active, STREAM);
  }
#define GO(NT, RG, KW) return out_f32 ? launch_rows<float, NT, RG, KW>(P, max_active, STREAM) : launch_rows<bf16_t, NT, RG, KW>(P, max_active, STREAM)
  if (narrow) {
    if (P.B <= 8) GO(1, 1, 8);
    if (P.B <= 32) GO(4, 1, 8);
    GO(8, 1, 8);
  }
  if (P.B <= 2) GO(1, 1, 8);
  if (P.B <= 8) GO(1, 2, 4);
  if (P.B <= 16) GO(2, 4, 2);
  if (P.B <= 32) GO(4, 8, 1);
  GO(8, 8, 1);
#undef GO
}

// all of one storage type
B200_API int b200_moe_combine(const void* h, int ld_h, const void* y, int ld_y, const void* ys, int ld_ys, const int* slot, const float* weight,
                              void* out, int ld_out, int T, int E, int top, int f32, void* stream) {
  if (T <= 0 || E <= 0 || top <= 0) return -1;
  const uintptr_t addr = reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(ys) | reinterpret_cast<uintptr_t>(out);
  const bool vec = !(addr & 15) && !((E | ld_h | ld_y | ld_ys | ld_out) & 7);
#define GO(T_, W) \
  launch_k(moe_combine_kernel<T_, W>, dim3(T), dim3(256), 0, STREAM, (const T_*)h, ld_h, (const T_*)y, ld_y, (const T_*)ys, ld_ys, slot, weight, (T_*)out, ld_out, E, top)
  if (f32) { if (vec) GO(float, 8); else GO(float, 1); }
  else { if (vec) GO(bf16_t, 8); else GO(bf16_t, 1); }
#undef GO
  return DONE;
}
