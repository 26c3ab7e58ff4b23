// Products that keep 32-bit results.
//
//  * b200_linear_f32: x (fp32 or bf16) times a bf16 weight, fp32 accumulation and output: the dense
//    linears of a model that is run in 32 bits. Plain FMA tiles, no reduced-precision mode.
//  * b200_router: router logits, scores and top-k of a mixture of experts in one kernel. The logits of
//    a block of tokens stay in shared memory as fp32, and one warp per token turns them into scores and
//    picks the experts. Few tokens: fp32 FMA with the token rows in shared memory, one expert per warp.
//    Many bf16 tokens: bf16 tensor-core products, which are exact, accumulated in fp32.
//    Group-limited choice (the best groups by the sum of their two best experts) happens in the same warp, and
//    a further weight row can give the sigmoid gate of a shared expert.
//  * b200_pair_linear_f32: one weight matrix per (token, choice) pair, the expert products of the
//    32-bit mode.
#include "common.cuh"
#include "mma_sync.cuh"

namespace b200 {

template <typename T>
__device__ __forceinline__ float to_f32(T v);
template <>
__device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

// ------------------------------------------------------------------------------------------
// dense
// ------------------------------------------------------------------------------------------
constexpr int kLT = 64, kLK = 16;

template <typename T>
__global__ void __launch_bounds__(256)
linear_f32_kernel(const T* __restrict__ x, const __nv_bfloat16* __restrict__ w, const __nv_bfloat16* __restrict__ bias,
                  float* __restrict__ out, int m, int n, int k, long long ldx, long long ldw, long long ldo, int act) {
  __shared__ float xs[kLK][kLT + 4], ws[kLK][kLT + 4];
  const int m0 = blockIdx.y * kLT, n0 = blockIdx.x * kLT;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < k; k0 += kLK) {
    for (int i = tid; i < kLT * kLK; i += 256) {
      const int r = i / kLK, c = i % kLK;
      xs[c][r] = (m0 + r < m && k0 + c < k) ? to_f32(x[(m0 + r) * ldx + k0 + c]) : 0.f;
      ws[c][r] = (n0 + r < n && k0 + c < k) ? __bfloat162float(w[(n0 + r) * ldw + k0 + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < kLK; ++c) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[c][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&ws[c][tx * 4]);
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
    const int r = m0 + ty * 4 + i;
    if (r >= m) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = n0 + tx * 4 + j;
      if (c < n) {
        const float v = acc[i][j] + (bias ? __bfloat162float(bias[c]) : 0.f);
        out[r * ldo + c] = act == 3 ? relu2(v) : (act & 255) == 4 && c >= act >> 8 ? tanhf(v) : v;
      }
    }
  }
}

// ------------------------------------------------------------------------------------------
// router
// ------------------------------------------------------------------------------------------
struct RouterParams {
  const void* x;               // [tokens][ldx]
  const __nv_bfloat16* w;      // [experts][ldw]
  const float* bias;           // [experts] added to the scores for the choice only (may be null)
  int* ids;                    // [tokens][top_k]
  float* wts;                  // [tokens][top_k]
  int tokens, experts, k, ldx, ldw, top_k, sigmoid, norm_topk;
  float scale;
  int n_group, topk_group;     // n_group > 1: only experts of the best topk_group groups of neighbours
  int rows;                    // weight rows: experts, and one more when gate is given
  float* gate;                 // [tokens] sigmoid of the last row's logit (may be null)
};

// Order-preserving map of a float to an unsigned integer (for warp-wide integer max)
__device__ __forceinline__ unsigned ordered_bits(float v) {
  const unsigned u = __float_as_uint(v);
  return (u >> 31) ? ~u : u | 0x80000000u;
}

// One warp: logits row [experts] in shared memory -> scores (in place), top-k by score + bias, ties to the
// lowest index. A chosen expert's score is stored with its sign bit set so that later rounds pass over it
// (scores are never negative).
__device__ __forceinline__ void route_row(float* row, const RouterParams& p, int t) {
  const int lane = threadIdx.x & 31;
  if (p.gate && lane == 0) p.gate[t] = 1.f / (1.f + expf(-row[p.experts]));
  if (p.sigmoid) {
    for (int e = lane; e < p.experts; e += 32) row[e] = 1.f / (1.f + expf(-row[e]));
  } else {
    float mx = -INFINITY;
    for (int e = lane; e < p.experts; e += 32) mx = fmaxf(mx, row[e]);
    mx = warp_max(mx);
    float s = 0.f;
    for (int e = lane; e < p.experts; e += 32) {
      const float v = expf(row[e] - mx);
      row[e] = v;
      s += v;
    }
    s = warp_sum(s);
    for (int e = lane; e < p.experts; e += 32) row[e] /= s;
  }
  if (p.n_group > 1 && p.topk_group < p.n_group) {
    // lane g ranks group g; experts of the other groups are passed over like chosen ones
    __syncwarp();
    const int size = p.experts / p.n_group;
    unsigned value = 0;
    if (lane < p.n_group) {
      float b1 = -INFINITY, b2 = -INFINITY;
      for (int e = lane * size; e < (lane + 1) * size; ++e) {
        const float s = row[e] + (p.bias ? p.bias[e] : 0.f);
        b2 = fmaxf(b2, fminf(b1, s));
        b1 = fmaxf(b1, s);
      }
      value = ordered_bits(size > 1 ? b1 + b2 : b1);
    }
    unsigned kept = 0;
    for (int r = 0; r < p.topk_group; ++r) {
      const unsigned v = (kept >> lane) & 1 ? 0u : value;
      const unsigned top = __reduce_max_sync(0xffffffffu, v);
      kept |= 1u << (__ffs(__ballot_sync(0xffffffffu, v == top)) - 1);
    }
    for (int e = lane; e < p.experts; e += 32)
      if (!((kept >> (e / size)) & 1)) row[e] = __uint_as_float(__float_as_uint(row[e]) | 0x80000000u);
    __syncwarp();
  }
  float wsum = 0.f, my_w = 0.f;
  int my_id = 0;
  for (int r = 0; r < p.top_k; ++r) {
    unsigned best = 0;
    int idx = 0x7fffffff;
    for (int e = lane; e < p.experts; e += 32) {
      const float s = row[e];
      if (__float_as_uint(s) >> 31) continue;
      const unsigned key = ordered_bits(s + (p.bias ? p.bias[e] : 0.f));
      if (key > best) { best = key; idx = e; }
    }
    const unsigned top = __reduce_max_sync(0xffffffffu, best);
    idx = __reduce_min_sync(0xffffffffu, best == top ? idx : 0x7fffffff);
    if (idx >= p.experts) idx = r < p.experts ? r : 0;      // only with scores that are not numbers
    const float raw = __uint_as_float(__float_as_uint(row[idx]) & 0x7fffffffu);
    __syncwarp();
    if (lane == 0) row[idx] = __uint_as_float(__float_as_uint(raw) | 0x80000000u);
    __syncwarp();
    if (lane == r) { my_w = raw; my_id = idx; }
    wsum += raw;
  }
  if (lane < p.top_k) {
    p.ids[static_cast<long long>(t) * p.top_k + lane] = my_id;
    p.wts[static_cast<long long>(t) * p.top_k + lane] = (p.norm_topk ? my_w / (wsum + 1e-20f) : my_w) * p.scale;
  }
}

// Few tokens (and the 32-bit mode): kTok tokens per block in shared memory as fp32, one expert per warp and
// turn. k is a multiple of 8. Dynamic shared memory: kTok * (k + rows) floats.
template <typename T, int kTok>
__global__ void __launch_bounds__(kTok > 2 ? 512 : 1024) router_kernel(const RouterParams p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float sm[];
  float* xs = sm;                       // [kTok][k]
  float* lg = sm + kTok * p.k;          // [kTok][rows]
  const int t0 = blockIdx.x * kTok;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
#pragma unroll
  for (int r = 0; r < kTok; ++r) {
    const T* xr = static_cast<const T*>(p.x) + static_cast<long long>(min(t0 + r, p.tokens - 1)) * p.ldx;
    for (int c = threadIdx.x; c < p.k; c += blockDim.x) xs[r * p.k + c] = to_f32(xr[c]);
  }
  __syncthreads();
  for (int e = warp; e < p.rows; e += warps) {
    float acc[kTok];
#pragma unroll
    for (int j = 0; j < kTok; ++j) acc[j] = 0.f;
    const __nv_bfloat16* wr = p.w + static_cast<long long>(e) * p.ldw;
#pragma unroll 4
    for (int c = lane * 8; c < p.k; c += 256) {
      const uint4 raw = *reinterpret_cast<const uint4*>(wr + c);
      const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&raw);
      float wv[8];
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 f = __bfloat1622float2(b[q]);
        wv[2 * q] = f.x;
        wv[2 * q + 1] = f.y;
      }
#pragma unroll
      for (int j = 0; j < kTok; ++j) {
        const float4 u = *reinterpret_cast<const float4*>(xs + j * p.k + c);
        const float4 v = *reinterpret_cast<const float4*>(xs + j * p.k + c + 4);
        acc[j] += u.x * wv[0] + u.y * wv[1] + u.z * wv[2] + u.w * wv[3];
        acc[j] += v.x * wv[4] + v.y * wv[5] + v.z * wv[6] + v.w * wv[7];
      }
    }
#pragma unroll
    for (int j = 0; j < kTok; ++j) {
      const float s = warp_sum(acc[j]);
      if (lane == 0) lg[j * p.rows + e] = s;
    }
  }
  __syncthreads();
  for (int j = warp; j < kTok; j += warps)
    if (t0 + j < p.tokens) route_row(lg + j * p.rows, p, t0 + j);
}

// Many bf16 tokens: 32 tokens per block, bf16 products with fp32 accumulation on the tensor core (m16n8k16),
// experts in passes of kRtExp. Warp (wm, wn): tokens 16 wm.., experts kRtExp / 2 wn.. of the pass. Dynamic shared
// memory: a ring of kRtStages stages of [32 + kRtExp] rows of 64 values (16-byte chunks XOR-swizzled by row),
// then 32 * rows floats.
constexpr int kRtTok = 32, kRtK = 64, kRtStages = 5;

template <int kRtExp>
__global__ void __launch_bounds__(128) router_tc_kernel(const RouterParams p) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(128) uint8_t smraw[];
  constexpr int kStage = (kRtTok + kRtExp) * kRtK * 2;
  float* lg = reinterpret_cast<float*>(smraw + kRtStages * kStage);
  constexpr int kNt = kRtExp / 16;                  // 8-wide expert tiles per warp
  const uint32_t base = smem_u32(smraw);
  const int t0 = blockIdx.x * kRtTok;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wm = warp & 1, wn = warp >> 1;
  const auto* x = static_cast<const __nv_bfloat16*>(p.x);
  const int nk = (p.k + kRtK - 1) / kRtK;
  for (int e0 = 0; e0 < p.rows; e0 += kRtExp) {
    auto load = [&](int kb, int st) {
      if (kb < nk) {
        for (int i = threadIdx.x; i < (kRtTok + kRtExp) * 8; i += 128) {
          const int r = i >> 3, c = i & 7, col = kb * kRtK + c * 8;
          const __nv_bfloat16* src = x;
          bool ok = col < p.k;
          if (r < kRtTok) {
            ok = ok && t0 + r < p.tokens;
            if (ok) src = x + static_cast<long long>(t0 + r) * p.ldx + col;
          } else {
            const int e = e0 + r - kRtTok;
            ok = ok && e < p.rows;
            if (ok) src = p.w + static_cast<long long>(e) * p.ldw + col;
          }
          cp_async_16(base + st * kStage + r * (kRtK * 2) + ((c ^ (r & 7)) << 4), src, ok);
        }
      }
      cp_async_commit();
    };
    float acc[kNt][4];
#pragma unroll
    for (int i = 0; i < kNt; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int i = 0; i < kRtStages - 1; ++i) load(i, i);
    int cur = 0;
    for (int kb = 0; kb < nk; ++kb) {
      cp_async_wait<kRtStages - 2>();
      __syncthreads();                              // stage kb has landed, stage kb - 1 has been read by all
      load(kb + kRtStages - 1, cur == 0 ? kRtStages - 1 : cur - 1);
      const uint32_t st = base + cur * kStage;
      cur = cur + 1 == kRtStages ? 0 : cur + 1;
#pragma unroll
      for (int kk = 0; kk < kRtK / 16; ++kk) {
        uint32_t a[4];
        const int ar = wm * 16 + (lane & 15), ac = kk * 2 + (lane >> 4);
        ldmatrix_x4(st + ar * (kRtK * 2) + ((ac ^ (ar & 7)) << 4), a[0], a[1], a[2], a[3]);
#pragma unroll
        for (int g = 0; g < kNt / 2; ++g) {
          const int mi = lane >> 3;
          const int br = kRtTok + wn * (kRtExp / 2) + g * 16 + (lane & 7) + 8 * (mi >> 1), bc = kk * 2 + (mi & 1);
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(st + br * (kRtK * 2) + ((bc ^ (br & 7)) << 4), b0, b1, b2, b3);
          mma_bf16_16816(acc[g * 2], a, b0, b1);
          mma_bf16_16816(acc[g * 2 + 1], a, b2, b3);
        }
      }
    }
    cp_async_wait<0>();
    __syncthreads();
    const int row = wm * 16 + (lane >> 2);
#pragma unroll
    for (int g = 0; g < kNt; ++g)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int e = e0 + wn * (kRtExp / 2) + g * 8 + (lane & 3) * 2 + (j & 1);
        if (e < p.rows) lg[(row + 8 * (j >> 1)) * p.rows + e] = acc[g][j];
      }
  }
  __syncthreads();
  for (int j = warp; j < kRtTok; j += 4)
    if (t0 + j < p.tokens) route_row(lg + j * p.rows, p, t0 + j);
}

template <typename T>
int launch_router(const RouterParams& p, bool tensor_cores, cudaStream_t stream) {
  const int limit = 200 * 1024;
  cudaError_t e;
  const int tile = p.rows <= 32 ? 32 : p.rows <= 64 ? 64 : p.rows <= 96 ? 96 : 128;
  const int tc_bytes = kRtStages * (kRtTok + tile) * kRtK * 2 + kRtTok * p.rows * 4;
  if (tensor_cores && p.tokens > 4 * 148 && tc_bytes <= limit && p.ldx % 8 == 0) {
    auto tc = [&](auto kernel, PerDeviceOnce& once) {
      if (once.first_time()) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, limit);
      return launch_pdl(kernel, dim3((p.tokens + kRtTok - 1) / kRtTok), dim3(128), tc_bytes, stream, p);
    };
    static PerDeviceOnce once_tc[4];
    switch (tile) {
      case 32: e = tc(router_tc_kernel<32>, once_tc[0]); break;
      case 64: e = tc(router_tc_kernel<64>, once_tc[1]); break;
      case 96: e = tc(router_tc_kernel<96>, once_tc[2]); break;
      default: e = tc(router_tc_kernel<128>, once_tc[3]); break;
    }
    return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
  }
  auto bytes = [&](int tok) { return tok * (p.k + p.rows) * 4; };
  // enough blocks to cover the machine first, then as many tokens per read of the weights as fit
  int tok = p.tokens >= 4 * 148 ? 8 : p.tokens >= 2 * 148 ? 4 : p.tokens > 148 ? 2 : 1;
  while (tok > 1 && bytes(tok) > limit / 2) tok /= 2;
  if (bytes(tok) > limit) return -2;
  const int threads = p.experts > 16 ? (tok > 2 ? 512 : 1024) : 512;
  auto go = [&](auto kernel, int n, PerDeviceOnce& once) {
    if (once.first_time()) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, limit);
    return launch_pdl(kernel, dim3((p.tokens + n - 1) / n), dim3(threads), bytes(n), stream, p);
  };
  static PerDeviceOnce once[4];
  switch (tok) {
    case 8: e = go(router_kernel<T, 8>, 8, once[3]); break;
    case 4: e = go(router_kernel<T, 4>, 4, once[2]); break;
    case 2: e = go(router_kernel<T, 2>, 2, once[1]); break;
    default: e = go(router_kernel<T, 1>, 1, once[0]); break;
  }
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

// out[pair][j] = x[pair / div] . w[ids[pair]][j] for ids below `experts` (other pairs are skipped).
// One warp per output feature, eight features per block.
__global__ void __launch_bounds__(256)
pair_linear_f32_kernel(const float* __restrict__ x, const __nv_bfloat16* __restrict__ w, const int* __restrict__ ids,
                       float* __restrict__ out, int div, int experts, int n, int k, long long ldx, long long ldo, int act) {
  const int pair = blockIdx.y, e = ids[pair];
  if (e < 0 || e >= experts) return;
  const int j = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (j >= n) return;
  const float* xr = x + static_cast<long long>(pair / div) * ldx;
  const __nv_bfloat16* wr = w + (static_cast<long long>(e) * n + j) * k;
  float s = 0.f;
  for (int c = lane; c < k; c += 32) s += xr[c] * __bfloat162float(wr[c]);
  s = warp_sum(s);
  if (lane == 0) out[static_cast<long long>(pair) * ldo + j] = act == 3 ? relu2(s) : s;
}

}  // namespace b200

using namespace b200;

// act: 0 none, 3 relu squared, 4 tanh of the output features from act >> 8 on
B200_API int b200_linear_f32(const void* x, int x_f32, const void* w, const void* bias, void* out, int m, int n, int k,
                             long long ldx, long long ldw, long long ldo, int act, cudaStream_t stream) {
  if (act != 0 && act != 3 && (act & 255) != 4) return -2;
  if (m <= 0 || n <= 0) return 0;
  const dim3 grid((n + kLT - 1) / kLT, (m + kLT - 1) / kLT);
  if (grid.y > 65535) return -2;
  const auto* wp = static_cast<const __nv_bfloat16*>(w);
  const auto* bp = static_cast<const __nv_bfloat16*>(bias);
  if (x_f32)
    linear_f32_kernel<float><<<grid, 256, 0, stream>>>(static_cast<const float*>(x), wp, bp, static_cast<float*>(out), m, n, k,
                                                       ldx, ldw, ldo, act);
  else
    linear_f32_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(static_cast<const __nv_bfloat16*>(x), wp, bp,
                                                               static_cast<float*>(out), m, n, k, ldx, ldw, ldo, act);
  return cudaGetLastError() == cudaSuccess ? 0 : -300;
}

// ids / wts [tokens][top_k] from x [tokens][k] (fp32 or bf16) and the router weight [experts][k] bf16:
// softmax or sigmoid scores in 32 bits, top-k by score + bias, weights = scores (optionally
// renormalised) * scale. k a multiple of 8, top_k <= 32. n_group > 1 (at most 32): group-limited choice. gate
// (may be null) [tokens]: sigmoid of the logit of one more weight row behind the experts'.
B200_API int b200_router(const void* x, int x_f32, const void* w, const float* bias, int* ids, float* wts, int tokens,
                         int experts, int k, int ldx, int ldw, int top_k, int sigmoid, int norm_topk, float scale,
                         int n_group, int topk_group, float* gate, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (k % 8 || ldw % 8 || top_k < 1 || top_k > 32 || top_k > experts) return -2;
  if (n_group > 1 && (n_group > 32 || experts % n_group || topk_group < 1 || topk_group > n_group)) return -2;
  RouterParams p{x, static_cast<const __nv_bfloat16*>(w), bias, ids, wts, tokens, experts, k, ldx, ldw, top_k, sigmoid,
                 norm_topk, scale, n_group, topk_group, experts + (gate ? 1 : 0), gate};
  return x_f32 ? launch_router<float>(p, false, stream) : launch_router<__nv_bfloat16>(p, true, stream);
}

B200_API int b200_pair_linear_f32(const void* x, const void* w, const int* ids, void* out, int pairs, int div, int experts,
                                  int n, int k, long long ldx, long long ldo, int act, cudaStream_t stream) {
  if (act != 0 && act != 3) return -2;
  if (pairs <= 0 || n <= 0) return 0;
  // the pair index is the grid's second dimension: run longer lists in slices (slices start on a token)
  const int step = 65535 / div * div;
  for (int p0 = 0; p0 < pairs; p0 += step) {
    const int cnt = pairs - p0 < step ? pairs - p0 : step;
    pair_linear_f32_kernel<<<dim3((n + 7) / 8, cnt), 256, 0, stream>>>(
        static_cast<const float*>(x) + static_cast<long long>(p0 / div) * ldx, static_cast<const __nv_bfloat16*>(w), ids + p0,
        static_cast<float*>(out) + static_cast<long long>(p0) * ldo, div, experts, n, k, ldx, ldo, act);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -300;
}
