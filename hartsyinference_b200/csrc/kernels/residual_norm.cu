// Norms around a 32-bit residual stream, and the embedding that starts it.
//
//   x  <- x + m * norm(y) * w_b              (sublayer output; left out for the first norm of a stack)
//   h  <- norm(x) * w_n                      (input of the next sublayer or of the output head; or x itself)
//
// in one launch per sublayer: the row stays in registers between the two norms, the stream is read
// and written once as fp32, y and h are in the activation type (bf16, or fp32 for a model run in
// 32 bits). y can also be given as routed expert rows: the weighted sum over the chosen experts
//   y[t] = sum_k w[t][k] * (slot_of[t][k] >= 0 ? rows[slot_of[t][k]] : ids[t][k] >= experts ? src[t] : 0)
// is formed in registers first (an expert index past the last real expert returns its input), so the
// combine step of a mixture of experts needs no launch and no intermediate rounding of its own; a shared expert's
// rows join the sum with one weight per token.
// LayerNorm (weight, no bias) or RMSNorm; weights as stored or stored around zero (1 + w); statistics in two
// passes over the registers, in fp32. An RMS norm on x can also be taken over equal parts of the row, each on its own,
// and at one token per sequence h can go through the convolutions over time that the next sublayers read
// (h + conv_i(h), see ssm.cu for prompts) in the same launch. The norm on x can also be tanh(alpha x) w + b, which has no statistics.
// cap_logits scales and caps the output logits; side_gate is the elementwise step of a second embedding that enters every layer. The embedding can be normed on its way into the stream, and poly_norm is
// the activation that mixes a row's normed powers.
#include "mixer_common.cuh"

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
  int plus_one;              // norms multiply by 1 + w
  int plain;                 // no w_n: h is the stream itself
  float eps, mult;           // mult: factor of the (normed) sublayer output
  const __nv_bfloat16* b_n;  // not null: h = tanh(alpha x) w_n + b_n
  float alpha;
  const void* extra;         // routed source: [rows][ld_extra] added with weight extra_w[row] (null: none)
  const float* extra_w;
  int ld_extra;
  int groups;                // > 1: w_n's norm is an RMS norm of this many equal parts
  const float* conv_w;       // not null: [conv_n][taps][ldh]; h is [conv_n][rows][ldh]
  int conv_n, taps;
  void* conv_state;          // [slots][taps - 1][ldh] earlier h, oldest first; moved on by one
  const int* positions;      // [rows], 0: the sequence starts
  const int* slots;          // [rows]
};

// v <- norm(v) * w over the row's first `dim` values (values past them are zero on entry and exit)
template <int kIters>
__device__ __forceinline__ void norm_row(float (&v)[kIters][8], const __nv_bfloat16* w, int dim, int layernorm,
                                         int plus_one, float eps, float* red) {
  const float one = plus_one ? 1.f : 0.f;
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
      for (int j = 0; j < 8; ++j) v[i][j] = (v[i][j] - mean) * inv * (one + wv[j]);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] = c + j < dim ? (v[i][j] - mean) * inv * (one + __bfloat162float(w[c + j])) : 0.f;
    }
  }
}

// v <- norm of each of `groups` equal parts of the row, times w. xr: the row as stored (this block's stores of it are
// done); sm: dim / 8 + groups floats of shared memory
template <int kIters>
__device__ __forceinline__ void group_norm_row(float (&v)[kIters][8], const float* xr, const __nv_bfloat16* w, int dim, int groups,
                                               int plus_one, float eps, float* sm) {
  const float one = plus_one ? 1.f : 0.f;
  const int n = dim / groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const bool whole = (n & 7) == 0;                 // parts consist of whole vectors
  float* inv = sm + (dim + 7) / 8;
  if (whole) {
#pragma unroll
    for (int i = 0; i < kIters; ++i) {
      const int vec = threadIdx.x + i * blockDim.x;
      float q = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) q = fmaf(v[i][j], v[i][j], q);
      if (vec * 8 < dim) sm[vec] = q;
    }
  }
  __syncthreads();
  for (int g = warp; g < groups; g += warps) {
    float q = 0.f;
    if (whole) for (int e = lane; e < n / 8; e += 32) q += sm[g * (n / 8) + e];
    else for (int e = lane; e < n; e += 32) q = fmaf(xr[g * n + e], xr[g * n + e], q);
    q = warp_sum(q);
    if (lane == 0) inv[g] = 1.f / sqrtf(q / n + eps);
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    if (c + 8 <= dim && whole) {
      float wv[8];
      load8(w + c, wv);
      const float f = inv[c / n];
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] = v[i][j] * f * (one + wv[j]);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] = c + j < dim ? v[i][j] * inv[(c + j) / n] * (one + __bfloat162float(w[c + j])) : 0.f;
    }
  }
}

// One token per sequence: h[i][row] = v + sum over the taps, the state moves on by one token. The state was last written
// by an earlier step, not by the kernel right before this one: up to three rows of it are read ahead of the wait.
constexpr int kConvAhead = 3;

template <typename T, int kIters>
struct ConvAhead {
  struct alignas(16) Vec { T v[8]; };       // as stored: half the registers for bf16
  Vec in[kIters][kConvAhead];
  __device__ __forceinline__ void load(const ResidualNormParams& p, long long row) {
    const int slot = p.slots[row], tail = p.taps - 1;
    const bool carried = slot >= 0 && p.positions[row] > 0;
    const T* state = static_cast<const T*>(p.conv_state) + static_cast<long long>(slot < 0 ? 0 : slot) * tail * p.ldh;
#pragma unroll
    for (int i = 0; i < kIters; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * 8;
#pragma unroll
      for (int k = 0; k < kConvAhead; ++k) {
        in[i][k] = Vec{};
        if (carried && k < tail && c < p.ldh) in[i][k] = *reinterpret_cast<const Vec*>(state + static_cast<long long>(k) * p.ldh + c);
      }
      if (c < p.ldh)                          // weights on their way into L2
        for (int k = 0; k < p.conv_n * p.taps; ++k) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.conv_w + static_cast<long long>(k) * p.ldh + c));
      if (p.w_n != nullptr && c < p.dim) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.w_n + c));
    }
  }
};

template <typename T, int kIters>
__device__ __forceinline__ void conv_row(const ResidualNormParams& p, long long row, const float (&v)[kIters][8], const ConvAhead<T, kIters>& ahead) {
  const int slot = p.slots[row], tail = p.taps - 1;
  const bool carried = slot >= 0 && p.positions[row] > 0;
  T* state = static_cast<T*>(p.conv_state) + static_cast<long long>(slot < 0 ? 0 : slot) * tail * p.ldh;
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    if (c >= p.ldh) continue;
    float now[8], y[2][8];
#pragma unroll
    for (int j = 0; j < 8; ++j) now[j] = y[0][j] = y[1][j] = ld1_of<T>(v[i][j]);
    auto tap = [&](int k, const float (&in)[8]) {
      if (k > 0 && slot >= 0) store8(state + static_cast<long long>(k - 1) * p.ldh + c, in);
#pragma unroll
      for (int o = 0; o < 2; ++o)
        if (o < p.conv_n) {
          float w[8];
          load8(p.conv_w + (static_cast<long long>(o) * p.taps + k) * p.ldh + c, w);
#pragma unroll
          for (int j = 0; j < 8; ++j) y[o][j] = fmaf(in[j], w[j], y[o][j]);
        }
    };
#pragma unroll
    for (int k = 0; k < kConvAhead; ++k)
      if (k < tail) {
        float in[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) in[j] = ld1(&ahead.in[i][k].v[j]);
        tap(k, in);
      }
    for (int k = kConvAhead; k < tail; ++k) {
      float in[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) in[j] = 0.f;
      if (carried) load8(state + static_cast<long long>(k) * p.ldh + c, in);
      tap(k, in);
    }
    tap(tail, now);
#pragma unroll
    for (int o = 0; o < 2; ++o)
      if (o < p.conv_n) store8(static_cast<T*>(p.h) + (static_cast<long long>(o) * gridDim.x + row) * p.ldh + c, y[o]);
  }
}

// v <- tanh(alpha v) * w + b over the row's first `dim` values, zero past them
template <int kIters>
__device__ __forceinline__ void tanh_row(float (&v)[kIters][8], const __nv_bfloat16* w, const __nv_bfloat16* b, float alpha, int dim) {
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    if (c + 8 <= dim) {
      float wv[8], bv[8];
      load8(w + c, wv);
      load8(b + c, bv);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[i][j] = fmaf(tanhf(alpha * v[i][j]), wv[j], bv[j]);
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j)
        v[i][j] = c + j < dim ? fmaf(tanhf(alpha * v[i][j]), __bfloat162float(w[c + j]), __bfloat162float(b[c + j])) : 0.f;
    }
  }
}

// One block per row; every leading dimension is a multiple of 8 and covers dim rounded up to 8.
// kConv: conv_w is given (rows come one per sequence, so they are few and two vectors per thread mean long ones).
template <typename T, int kIters, bool kConv>
__global__ void __launch_bounds__(1024) residual_norm_kernel(const ResidualNormParams p) {
  const long long row = blockIdx.x;
  ConvAhead<T, kConv ? kIters : 1> ahead;
  if (kConv) ahead.load(p, row);
  pdl_wait();
  pdl_trigger();
  __shared__ float red[32];
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
      if (p.extra != nullptr) {
        const T* sp = static_cast<const T*>(p.extra) + row * p.ld_extra;
        const float w = p.extra_w[row];
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
    if (p.w_b != nullptr) norm_row<kIters>(yv, p.w_b, p.dim, p.layernorm, p.plus_one, p.eps, red);
#pragma unroll
    for (int i = 0; i < kIters; ++i) {
      const int c = (threadIdx.x + i * blockDim.x) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j) xv[i][j] = 0.f;
      if (c < p.dim) {
        load8(xr + c, xv[i]);
#pragma unroll
        for (int j = 0; j < 8; ++j) xv[i][j] = fmaf(p.mult, yv[i][j], xv[i][j]);
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
  if (p.w_n == nullptr && !p.plain) return;
  if (p.b_n != nullptr) tanh_row<kIters>(xv, p.w_n, p.b_n, p.alpha, p.dim);
  else if (p.w_n != nullptr && p.groups > 1) {
    extern __shared__ float parts[];
    group_norm_row<kIters>(xv, xr, p.w_n, p.dim, p.groups, p.plus_one, p.eps, parts);
  } else if (p.w_n != nullptr) norm_row<kIters>(xv, p.w_n, p.dim, p.layernorm, p.plus_one, p.eps, red);
  if constexpr (kConv) {
    conv_row<T, kIters>(p, row, xv, ahead);
    return;
  }
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

// x[t] = norm(table[id]) * w in fp32 (the stream) and h[t] = x[t] in the activation type. ids null: the rows of
// `table` in order.
struct EmbeddingNormParams {
  const int* ids;
  const __nv_bfloat16* table;
  const __nv_bfloat16* w;
  float* x;
  void* h;
  int dim, ldx, ldt, vocab, layernorm, plus_one;
  float scale, eps;
};

template <typename T, int kIters>
__global__ void __launch_bounds__(1024) embedding_norm_kernel(const EmbeddingNormParams p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[32];
  const long long t = blockIdx.x;
  long long id = t;
  if (p.ids) id = min(max(p.ids[t], 0), p.vocab - 1);
  const __nv_bfloat16* src = p.table + id * p.ldt;
  float v[kIters][8];
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[i][j] = 0.f;
    if (c < p.dim) load8(src + c, v[i]);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[i][j] = c + j < p.dim ? v[i][j] * p.scale : 0.f;
  }
  norm_row<kIters>(v, p.w, p.dim, p.layernorm, p.plus_one, p.eps, red);
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    if (c < p.ldx) {
      store8(p.x + t * p.ldx + c, v[i]);
      store8(static_cast<T*>(p.h) + t * p.ldx + c, v[i]);
    }
  }
}

// y[t][c] = gelu_tanh(u[t][c]) * table[ids[t]][off + c], eight values per thread
template <typename T>
__global__ void __launch_bounds__(256) side_gate_kernel(const T* __restrict__ u, const int* __restrict__ ids,
                                                        const __nv_bfloat16* __restrict__ table, T* __restrict__ y, long long n,
                                                        int vecs, int ldu, int ldt, int vocab) {
  pdl_wait();
  pdl_trigger();
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const long long t = i / vecs;
  const int c = static_cast<int>(i % vecs) * 8;
  const int id = min(max(ids[t], 0), vocab - 1);
  float a[8], e[8];
  load8(u + t * ldu + c, a);
  load8(table + static_cast<long long>(id) * ldt + c, e);
#pragma unroll
  for (int j = 0; j < 8; ++j) a[j] = gelu_tanh(a[j]) * e[j];
  store8(y + t * vecs * 8 + c, a);
}

// out = cap * tanh(scale y / cap), or scale y without a cap: logits in 32 bits. Eight values per thread.
template <typename T>
__global__ void __launch_bounds__(256) cap_logits_kernel(const T* __restrict__ y, float* __restrict__ out, long long n, float scale, float cap) {
  pdl_wait();
  pdl_trigger();
  const long long i = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) * 8;
  if (i >= n) return;
  const float inner = cap > 0.f ? scale / cap : scale;
  float v[8];
  if (i + 8 <= n) {
    load8(y + i, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = cap > 0.f ? cap * tanhf(v[j] * inner) : v[j] * inner;
    store8(out + i, v);
  } else {
    for (long long j = i; j < n; ++j) out[j] = cap > 0.f ? cap * tanhf(ld1(y + j) * inner) : ld1(y + j) * inner;
  }
}

// y = a z / rms(z) + b z^2 / rms(z^2) + c z^3 / rms(z^3) + e over a row of `dim` values (powers element by
// element); columns past dim are zeroed. The row stays in registers between the two passes.
template <typename T, int kIters>
__global__ void __launch_bounds__(512) poly_norm_kernel(const T* __restrict__ z, T* __restrict__ y,
                                                        const float* __restrict__ coef, int dim, int ldz, int ldy, float eps) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[3][16];
  struct alignas(16) Vec { T v[8]; };
  const long long row = blockIdx.x;
  Vec raw[kIters];                           // as stored: half the registers for bf16
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    raw[i] = Vec{};
    if (c < dim) raw[i] = *reinterpret_cast<const Vec*>(z + row * ldz + c);
  }
  float q1 = 0.f, q2 = 0.f, q3 = 0.f;
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float u = c + j < dim ? ld1(&raw[i].v[j]) : 0.f, s = u * u;
      q1 += s;
      q2 = fmaf(s, s, q2);
      q3 = fmaf(s * s, s, q3);
    }
  }
  q1 = warp_sum(q1);
  q2 = warp_sum(q2);
  q3 = warp_sum(q3);
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = q1;
    red[1][threadIdx.x >> 5] = q2;
    red[2][threadIdx.x >> 5] = q3;
  }
  __syncthreads();
  q1 = q2 = q3 = 0.f;
  for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) {
    q1 += red[0][i];
    q2 += red[1][i];
    q3 += red[2][i];
  }
  const float a = coef[0] / sqrtf(q1 / dim + eps), b = coef[1] / sqrtf(q2 / dim + eps), c3 = coef[2] / sqrtf(q3 / dim + eps);
  const float e = coef[3];
#pragma unroll
  for (int i = 0; i < kIters; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    if (c >= ldy) continue;
    float o[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float u = ld1(&raw[i].v[j]);
      o[j] = c + j < dim ? fmaf(u, fmaf(u, fmaf(u, c3, b), a), e) : 0.f;
    }
    store8(y + row * ldy + c, o);
  }
}

// Rows of up to 16384 values, eight per thread and vector: two vectors per thread for long rows, and when there
// are many rows (more bytes in flight per thread).
inline bool row_shape(int dim, int rows, int& iters, int& threads) {
  const int vecs = (dim + 7) / 8;
  iters = vecs > 1024 || (rows >= 1024 && vecs >= 128) ? 2 : 1;
  threads = ((vecs + iters - 1) / iters + 31) / 32 * 32;
  return threads <= 1024;
}

template <typename T>
int launch_residual_norm(const ResidualNormParams& p, int rows, cudaStream_t stream) {
  int iters, threads;
  if (!row_shape(p.dim, rows, iters, threads)) return -2;
  const int smem = p.groups > 1 ? ((p.dim + 7) / 8 + p.groups) * 4 : 0;
  auto go = [&](auto kernel) { return launch_pdl(kernel, dim3(rows), dim3(threads), smem, stream, p); };
  const cudaError_t e = p.conv_w ? (iters == 1 ? go(residual_norm_kernel<T, 1, true>) : go(residual_norm_kernel<T, 2, true>))
                                 : (iters == 1 ? go(residual_norm_kernel<T, 1, false>) : go(residual_norm_kernel<T, 2, false>));
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

}  // namespace b200

using namespace b200;

// See the header comment. f32 != 0: y / src / extra / h are fp32 instead of bf16. ldy etc. in elements,
// multiples of 8. Rows of at most 16384 values, norms of at most 2048 parts. conv_w (may be null): one or two sets of
// taps for h, one token per sequence.
B200_API int b200_residual_norm(void* x, const void* y, void* h, const void* w_b, const void* w_n, const int* slot_of,
                                const int* ids, const float* wts, const void* src, int rows, int dim, int ldx, int ldy,
                                int ldh, int ld_src, int top_k, int experts, int layernorm, int plus_one, int plain, float eps,
                                float mult, int f32, const void* b_n, float alpha, const void* extra, const float* extra_w,
                                int ld_extra, int groups, const float* conv_w, int conv_n, int taps, void* conv_state,
                                const int* positions, const int* slots, cudaStream_t stream) {
  if (rows <= 0) return 0;
  const int dim8 = (dim + 7) / 8 * 8;
  if (dim < 1 || dim > 16384 || ldx < dim8 || ldx % 8 || ((w_n || plain) && (ldh != dim8 || !h))) return -2;
  if (y && (ldy < dim8 || ldy % 8)) return -2;
  if (slot_of && (!ids || !wts || top_k < 1 || (src && (ld_src < dim8 || ld_src % 8)))) return -2;
  if ((b_n && !w_n) || (extra && (!slot_of || !extra_w || ld_extra < dim8 || ld_extra % 8))) return -2;
  if (groups > 1 && (groups > 2048 || dim % groups || layernorm || b_n)) return -2;
  if (conv_w && (conv_n < 1 || conv_n > 2 || taps < 1 || (taps > 1 && !conv_state) || !positions || !slots || !h)) return -2;
  ResidualNormParams p{static_cast<float*>(x), y, h, static_cast<const __nv_bfloat16*>(w_b),
                       static_cast<const __nv_bfloat16*>(w_n), slot_of, ids, wts, src, dim, ldx, ldy, ldh, ld_src, top_k,
                       experts, layernorm, plus_one, plain, eps, mult, static_cast<const __nv_bfloat16*>(b_n), alpha, extra, extra_w,
                       ld_extra, groups, conv_w, conv_n, taps, conv_state, positions, slots};
  return f32 ? launch_residual_norm<float>(p, rows, stream) : launch_residual_norm<__nv_bfloat16>(p, rows, stream);
}

// y [tokens][dim] from u [tokens][ldu] and rows of table [vocab][ldt] (already moved to the layer's columns); dim and
// both pitches multiples of 8
B200_API int b200_side_gate(const void* u, const int* ids, const void* table, void* y, int tokens, int dim, int ldu, int ldt,
                            int vocab, int f32, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (dim < 8 || dim % 8 || ldu % 8 || ldt % 8) return -2;
  const long long n = static_cast<long long>(tokens) * (dim / 8);
  const dim3 grid(static_cast<unsigned>((n + 255) / 256));
  const auto* tab = static_cast<const __nv_bfloat16*>(table);
  const cudaError_t e =
      f32 ? launch_pdl(side_gate_kernel<float>, grid, dim3(256), 0, stream, static_cast<const float*>(u), ids, tab,
                       static_cast<float*>(y), n, dim / 8, ldu, ldt, vocab)
          : launch_pdl(side_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, static_cast<const __nv_bfloat16*>(u), ids, tab,
                       static_cast<__nv_bfloat16*>(y), n, dim / 8, ldu, ldt, vocab);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

// out [n] fp32 from y [n] (fp32 or bf16); cap 0: scale only
B200_API int b200_cap_logits(const void* y, void* out, long long n, float scale, float cap, int f32, cudaStream_t stream) {
  if (n <= 0) return 0;
  const dim3 grid(static_cast<unsigned>((n + 2047) / 2048));
  const cudaError_t e = f32 ? launch_pdl(cap_logits_kernel<float>, grid, dim3(256), 0, stream, static_cast<const float*>(y),
                                         static_cast<float*>(out), n, scale, cap)
                            : launch_pdl(cap_logits_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, static_cast<const __nv_bfloat16*>(y),
                                         static_cast<float*>(out), n, scale, cap);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
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

// x fp32 and h (activation type) [tokens][ldx] = norm(table[ids] * scale) * w
B200_API int b200_embedding_norm(const int* ids, const void* table, const void* w, void* x, void* h, int tokens, int dim,
                                 int ldx, int ldt, int vocab, float scale, int layernorm, int plus_one, float eps, int f32,
                                 cudaStream_t stream) {
  if (tokens <= 0) return 0;
  int iters, threads;
  if (ldx % 8 || ldt % 8 || ldx != (dim + 7) / 8 * 8 || ldt < ldx || !row_shape(dim, tokens, iters, threads)) return -2;
  EmbeddingNormParams p{ids, static_cast<const __nv_bfloat16*>(table), static_cast<const __nv_bfloat16*>(w),
                        static_cast<float*>(x), h, dim, ldx, ldt, vocab, layernorm, plus_one, scale, eps};
  cudaError_t e;
  if (f32) e = iters == 1 ? launch_pdl(embedding_norm_kernel<float, 1>, dim3(tokens), dim3(threads), 0, stream, p)
                          : launch_pdl(embedding_norm_kernel<float, 2>, dim3(tokens), dim3(threads), 0, stream, p);
  else e = iters == 1 ? launch_pdl(embedding_norm_kernel<__nv_bfloat16, 1>, dim3(tokens), dim3(threads), 0, stream, p)
                      : launch_pdl(embedding_norm_kernel<__nv_bfloat16, 2>, dim3(tokens), dim3(threads), 0, stream, p);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

// y [rows][ldy] from z [rows][ldz]; coef: the four numbers a, b, c, e (fp32, device). Rows of up to 16384 values: one,
// two or four vectors of eight per thread.
B200_API int b200_poly_norm(const void* z, void* y, const float* coef, int rows, int dim, int ldz, int ldy, float eps, int f32,
                            cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (dim < 1 || dim > 16384 || ldz % 8 || ldy != (dim + 7) / 8 * 8 || ldz < ldy) return -2;
  const int vecs = ldy / 8;
  const int iters = vecs > 1024 || (rows >= 1024 && vecs >= 512) ? 4 : vecs > 512 || (rows >= 1024 && vecs >= 128) ? 2 : 1;
  const int threads = ((vecs + iters - 1) / iters + 31) / 32 * 32;
  auto go = [&](auto kernel, auto tag) {
    using T = decltype(tag);
    return launch_pdl(kernel, dim3(rows), dim3(threads), 0, stream, static_cast<const T*>(z), static_cast<T*>(y), coef, dim, ldz,
                      ldy, eps);
  };
  cudaError_t e;
  if (f32) e = iters == 1 ? go(poly_norm_kernel<float, 1>, float()) : iters == 2 ? go(poly_norm_kernel<float, 2>, float()) : go(poly_norm_kernel<float, 4>, float());
  else e = iters == 1 ? go(poly_norm_kernel<__nv_bfloat16, 1>, __nv_bfloat16()) : iters == 2 ? go(poly_norm_kernel<__nv_bfloat16, 2>, __nv_bfloat16())
                                                                                       : go(poly_norm_kernel<__nv_bfloat16, 4>, __nv_bfloat16());
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}
