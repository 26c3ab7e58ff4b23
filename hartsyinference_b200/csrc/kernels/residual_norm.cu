// Norms around a 32-bit residual stream, and the embedding that starts it.
//
//   x  <- x + norm(y) * w_b                  (sublayer output; left out for the first norm of a stack)
//   h  <- norm(x) * w_n                      (input of the next sublayer or of the output head)
//
// in one launch per sublayer: the row stays in registers between the two norms, the stream is read
// and written once as fp32, y and h are in the activation type (bf16, or fp32 for a model run in
// 32 bits). y can also be given as routed expert rows: the weighted sum over the chosen experts
//   y[t] = sum_k w[t][k] * (slot_of[t][k] >= 0 ? rows[slot_of[t][k]] : ids[t][k] >= experts ? src[t] : 0)
// is formed in registers first (an expert index past the last real expert returns its input), so the
// combine step of a mixture of experts needs no launch and no intermediate rounding of its own.
// LayerNorm (weight, no bias) or RMSNorm; statistics in two passes over the registers, in fp32.
#include "common.cuh"

namespace b200 {

struct ResidualNormParams {
  float* x;                  // [rows][ldx] residual stream, updated in place when y is given
  const void* y;             // [rows][ldy] sublayer output (or expert rows [slots][ldy]); null: norm only
  void* h;                   // [rows][ldh] normed output, columns dim..ldh are zeroed
  const __nv_bfloat16* w_b;  // [dim] weight of the norm on y (null: y is added as it is)
  const __nv_bfloat16* w_n;  // [dim] weight of the norm on x (null: no output)
  const int* slot_of;        // routed source: [rows][top_k]
  const int* ids;            //                [rows][top_k]
  const float* wts;          //                [rows][top_k]
  const void* src;           //                [rows][ld_src] what a pass-through expert returns
  int dim, ldx, ldy, ldh, ld_src, top_k, experts, layernorm;
  float eps;
};

template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <>
__device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = __bfloat1622float2(b[i]);
    v[2 * i] = f.x;
    v[2 * i + 1] = f.y;
  }
}
template <>
__device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <typename T>
__device__ __forceinline__ void store8(T* p, const float (&v)[8]);
template <>
__device__ __forceinline__ void store8<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 o;
  o.x = pack_bf16x2(v[0], v[1]);
  o.y = pack_bf16x2(v[2], v[3]);
  o.z = pack_bf16x2(v[4], v[5]);
  o.w = pack_bf16x2(v[6], v[7]);
  *reinterpret_cast<uint4*>(p) = o;
}
template <>
__device__ __forceinline__ void store8<float>(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  const int n = blockDim.x >> 5;
  float s = 0.f;
  for (int i = 0; i < n; ++i) s += red[i];
  return s;
}

// v <- norm(v) * w over the row's first `dim` values (values past them are zero on entry and exit)
template <int kIters>
__device__ __forceinline__ void norm_row(float (&v)[kIters][8], const __nv_bfloat16* w, int dim, int layernorm,
                                         float eps, float* red) {
  float mean = 0.f;
  if (layernorm) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < kIters; ++i)
#pragma unroll
      for (int j = 0; j < 8; ++j) s += v[i][j];
    mean = block_sum(s, red) / dim;
  }
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float d = c + j < dim ? v[i][j] - mean : 0.f;
      q += d * d;
    }
  }
  const float inv = 1.f / sqrtf(block_sum(q, red) / dim + eps);
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    if (c + 8 <= dim) {
      float wv[8];
      load8(w + c, wv);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] = (v[i][j] - mean) * inv * wv[j];
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] = c + j < dim ? (v[i][j] - mean) * inv * __bfloat162float(w[c + j]) : 0.f;
    }
  }
}

// One block per row; every leading dimension is a multiple of 8 and covers dim rounded up to 8.
template <typename T, int kIters>
__global__ void __launch_bounds__(1024) residual_norm_kernel(const ResidualNormParams p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[32];
  const long long row = blockIdx.x;
  float* xr = p.x + row * p.ldx;
  float xv[kIters][8];
  if (p.y != nullptr) {
    float yv[kIters][8];
#pragma unroll
    for (int i = 0; i < kIters; ++i)
#pragma unroll
      for (int j = 0; j < 8; ++j) yv[i][j] = 0.f;
    if (p.slot_of != nullptr) {
      for (int k = 0; k < p.top_k; ++k) {
        const int slot = p.slot_of[row * p.top_k + k];
        const T* sp = nullptr;
        if (slot >= 0) sp = static_cast<const T*>(p.y) + static_cast<long long>(slot) * p.ldy;
        else if (p.src != nullptr && p.ids[row * p.top_k + k] >= p.experts) sp = static_cast<const T*>(p.src) + row * p.ld_src;
        if (sp == nullptr) continue;
        const float w = p.wts[row * p.top_k + k];
#pragma unroll
        for (int i = 0; i < kIters; ++i) {
          const int c = (threadIdx.x + i * blockDim.x) * 8;
          if (c < p.dim) {
            float t[8];
            load8(sp + c, t);
#pragma unroll
            for (int j = 0; j < 8; ++j) yv[i][j] += w * t[j];
          }
        }
      }
    } else {
      const T* sp = static_cast<const T*>(p.y) + row * p.ldy;
#pragma unroll
      for (int i = 0; i < kIters; ++i) {
        const int c = (threadIdx.x + i * blockDim.x) * 8;
        if (c < p.dim) load8(sp + c, yv[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < kIters; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (c + j >= p.dim) yv[i][j] = 0.f;
    }
    if (p.w_b != nullptr) norm_row<kIters>(yv, p.w_b, p.dim, p.layernorm, p.eps, red);
#pragma unroll
    for (int i = 0; i < kIters; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j) xv[i][j] = 0.f;
      if (c < p.dim) {
        load8(xr + c, xv[i]);
#pragma unroll
        for (int j = 0; j < 8; ++j) xv[i][j] += yv[i][j];
        store8(xr + c, xv[i]);
      }
    }
  } else {
#pragma unroll
    for (int i = 0; i < kIters; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j) xv[i][j] = 0.f;
      if (c < p.dim) load8(xr + c, xv[i]);
    }
  }
  if (p.w_n == nullptr) return;
  norm_row<kIters>(xv, p.w_n, p.dim, p.layernorm, p.eps, red);
  T* hr = static_cast<T*>(p.h) + row * p.ldh;
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    if (c < p.ldh) store8(hr + c, xv[i]);
  }
}

// x[t] = table[id] * scale as fp32, columns dim..ldx zeroed
__global__ void embedding_f32_kernel(const int* __restrict__ ids, const __nv_bfloat16* __restrict__ table,
                                     float* __restrict__ x, int dim, int ldx, int ldt, int vocab, float scale) {
  const int t = blockIdx.x;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const __nv_bfloat16* src = table + static_cast<long long>(id) * ldt;
  float* dst = x + static_cast<long long>(t) * ldx;
  for (int c = threadIdx.x * 8; c < ldx; c += blockDim.x * 8) {
    float v[8];
    load8(src + c, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = c + j < dim ? v[j] * scale : 0.f;
    store8(dst + c, v);
  }
}

template <typename T>
int launch_residual_norm(const ResidualNormParams& p, int rows, cudaStream_t stream) {
  const int vecs = (p.dim + 7) / 8;
  // two vectors per thread for long rows, and when there are many rows (more bytes in flight per thread)
  const int iters = vecs > 1024 || (rows >= 1024 && vecs >= 128) ? 2 : 1;
  int threads = ((vecs + iters - 1) / iters + 31) / 32 * 32;
  if (threads > 1024) return -2;
  cudaError_t e;
  switch (iters) {
    case 1: e = launch_pdl(residual_norm_kernel<T, 1>, dim3(rows), dim3(threads), 0, stream, p); break;
    default: e = launch_pdl(residual_norm_kernel<T, 2>, dim3(rows), dim3(threads), 0, stream, p); break;
  }
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

}  // namespace b200

using namespace b200;

// See the header comment. f32 != 0: y / src / h are fp32 instead of bf16. ldy etc. in elements,
// multiples of 8. Rows of at most 16384 values.
B200_API int b200_residual_norm(void* x, const void* y, void* h, const void* w_b, const void* w_n, const int* slot_of,
                                const int* ids, const float* wts, const void* src, int rows, int dim, int ldx, int ldy,
                                int ldh, int ld_src, int top_k, int experts, int layernorm, float eps, int f32,
                                cudaStream_t stream) {
  if (rows <= 0) return 0;
  const int dim8 = (dim + 7) / 8 * 8;
  if (dim < 1 || dim > 16384 || ldx < dim8 || ldx % 8 || (w_n && (ldh != dim8 || !h))) return -2;
  if (y && (ldy < dim8 || ldy % 8)) return -2;
  if (slot_of && (!ids || !wts || top_k < 1 || (src && (ld_src < dim8 || ld_src % 8)))) return -2;
  ResidualNormParams p{static_cast<float*>(x), y, h, static_cast<const __nv_bfloat16*>(w_b),
                       static_cast<const __nv_bfloat16*>(w_n), slot_of, ids, wts, src, dim, ldx, ldy, ldh, ld_src, top_k,
                       experts, layernorm, eps};
  return f32 ? launch_residual_norm<float>(p, rows, stream) : launch_residual_norm<__nv_bfloat16>(p, rows, stream);
}

B200_API int b200_embedding_f32(const int* ids, const void* table, void* x, int tokens, int dim, int ldx, int ldt,
                                int vocab, float scale, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (ldx % 8 || ldt % 8 || ldx < dim || ldt < ldx) return -2;
  int threads = (ldx / 8 + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  embedding_f32_kernel<<<tokens, threads, 0, stream>>>(ids, static_cast<const __nv_bfloat16*>(table), static_cast<float*>(x),
                                                       dim, ldx, ldt, vocab, scale);
  return cudaGetLastError() == cudaSuccess ? 0 : -300;
}
