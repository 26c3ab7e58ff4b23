// Rotation of queries and keys for models with per-layer mixers, in 32 bits.
//
//  * rope_table       cosines and sines of every (token, frequency), once per batch and rotation for all layers. A
//                     frequency comes as the sum of two floats and the product with the position keeps its rounding
//                     error, so the angle is good to the last bit of the sine at any position.
//  * qk_rope_store    between the projection and attention, one launch: RMS norm of q and of k over all their heads
//                     at once (optional), rotation of the leading values of each head (optional, either pairing), q to a
//                     dense matrix, k and v straight into their pages. One block per token; the row is read twice, the
//                     second time from L1.
//  * head_norm_store  the same with a norm of every head on its own; k and v can be left out (a layer that reads another
//                     one's pages).
#include "mixer_common.cuh"

namespace b200 {

__global__ void __launch_bounds__(256) rope_table_kernel(const int* __restrict__ positions, const float* __restrict__ hi,
                                                         const float* __restrict__ lo, float2* __restrict__ out, long long n, int pairs) {
  pdl_wait();
  pdl_trigger();
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const long long t = i / pairs;
  const int j = static_cast<int>(i - t * pairs);
  const float pos = static_cast<float>(positions[t]);
  const float a = pos * hi[j], rest = fmaf(pos, hi[j], -a) + pos * lo[j];
  float s, c, rs, rc;
  sincosf(a, &s, &c);
  sincosf(rest, &rs, &rc);
  out[i] = make_float2(c * rc - s * rs, s * rc + c * rs);
}

struct QkRopeParams {
  const void* p;                 // [T][ld]: q heads at 0, k heads at k_off, v heads at v_off
  const __nv_bfloat16 *wq, *wk;  // [heads * d], [hkv * d] or null
  const float2* table;           // [T][rot / 2] or null
  void *q_out, *k_cache, *v_cache;
  const long long* slots;        // [T], < 0: not stored
  long long ld;
  int heads, hkv, d, dv, k_off, v_off, page;
  int rot, interleaved;
  float inv_q, inv_k;            // 1 / number of true values of q and of k
  float eps;
};

// Eight values from column c of a head: norm and rotation. x: the head's row, w: its weights or null.
template <typename T>
__device__ __forceinline__ void turned8(const QkRopeParams& p, const T* x, const __nv_bfloat16* w, float inv, const float2* cs, int c,
                                        float (&v)[8]) {
  load8(x + c, v);
  if (w) {
    float wv[8];
    load8(w + c, wv);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = v[j] * inv * wv[j];
  }
  if (!cs || c >= p.rot) return;
  const int half = p.rot >> 1;
  if (p.interleaved) {
#pragma unroll
    for (int j = 0; j < 8; j += 2)
      if (c + j < p.rot) {
        const float2 f = cs[(c + j) >> 1];
        const float a = v[j], b = v[j + 1];
        v[j] = a * f.x - b * f.y;
        v[j + 1] = b * f.x + a * f.y;
      }
    return;
  }
  float u[8];
  if ((half & 7) == 0) {                     // partners are one vector
    const int q = c < half ? c + half : c - half;
    load8(x + q, u);
    if (w) {
      float wv[8];
      load8(w + q, wv);
#pragma unroll
      for (int j = 0; j < 8; ++j) u[j] = u[j] * inv * wv[j];
    }
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int e = c + j, q = e < half ? e + half : e - half;
      u[j] = e < p.rot ? ld1(x + q) * (w ? inv * __bfloat162float(w[q]) : 1.f) : 0.f;
    }
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int e = c + j;
    if (e >= p.rot) continue;
    const float2 f = cs[e < half ? e : e - half];
    v[j] = e < half ? v[j] * f.x - u[j] * f.y : v[j] * f.x + u[j] * f.y;
  }
}

template <typename T>
__global__ void __launch_bounds__(512) qk_rope_store_kernel(const QkRopeParams p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[2][16];
  const long long t = blockIdx.x;
  const T* row = static_cast<const T*>(p.p) + t * p.ld;
  const int dvec = p.d >> 3, vvec = p.dv >> 3;
  const int nq = p.heads * dvec, nk = p.hkv * dvec, nv = p.hkv * vvec;
  float inv_q = 1.f, inv_k = 1.f;
  if (p.wq || p.wk) {
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
      float v[8], s = 0.f;
      load8(i < nq ? row + i * 8 : row + p.k_off + (i - nq) * 8, v);
#pragma unroll
      for (int j = 0; j < 8; ++j) s = fmaf(v[j], v[j], s);
      if (i < nq) sq += s; else sk += s;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) {
      red[0][threadIdx.x >> 5] = sq;
      red[1][threadIdx.x >> 5] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
    for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) {
      sq += red[0][i];
      sk += red[1][i];
    }
    inv_q = 1.f / sqrtf(sq * p.inv_q + p.eps);
    inv_k = 1.f / sqrtf(sk * p.inv_k + p.eps);
  }
  const float2* cs = p.table ? p.table + t * (p.rot >> 1) : nullptr;
  const long long slot = p.slots[t];
  const long long page = slot >= 0 ? slot / p.page : 0, off = slot >= 0 ? slot % p.page : 0;
  T* qo = static_cast<T*>(p.q_out) + t * p.heads * p.d;
  for (int i = threadIdx.x; i < nq + nk + nv; i += blockDim.x) {
    float v[8];
    if (i < nq) {
      const int h = i / dvec, c = (i - h * dvec) * 8;
      turned8(p, row + h * p.d, p.wq ? p.wq + h * p.d : nullptr, inv_q, cs, c, v);
      store8(qo + h * p.d + c, v);
    } else if (slot < 0) {
      break;
    } else if (i < nq + nk) {
      const int h = (i - nq) / dvec, c = (i - nq - h * dvec) * 8;
      turned8(p, row + p.k_off + h * p.d, p.wk ? p.wk + h * p.d : nullptr, inv_k, cs, c, v);
      store8(static_cast<T*>(p.k_cache) + ((page * p.hkv + h) * p.page + off) * p.d + c, v);
    } else {
      const int h = (i - nq - nk) / vvec, c = (i - nq - nk - h * vvec) * 8;
      load8(row + p.v_off + h * p.dv + c, v);
      store8(static_cast<T*>(p.v_cache) + ((page * p.hkv + h) * p.page + off) * p.dv + c, v);
    }
  }
}

// kLanes neighbouring lanes per head. p.inv_q: 1 / true head size; p.hkv 0: no keys and values.
template <typename T, int kLanes>
__global__ void __launch_bounds__(512) head_norm_store_kernel(const QkRopeParams p) {
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const T* row = static_cast<const T*>(p.p) + t * p.ld;
  const float2* cs = p.table ? p.table + t * (p.rot >> 1) : nullptr;
  const long long slot = p.slots[t];
  const long long page = slot >= 0 ? slot / p.page : 0, off = slot >= 0 ? slot % p.page : 0;
  const int g = threadIdx.x / kLanes, lane = threadIdx.x % kLanes, all = p.heads + p.hkv;
  for (int h0 = 0; h0 < all; h0 += blockDim.x / kLanes) {
    const int h = h0 + g;
    const bool is_q = h < p.heads, on = is_q || (h < all && slot >= 0);
    const T* x = row + (is_q ? h * p.d : p.k_off + (h - p.heads) * p.d);
    float s = 0.f;
    if (on)
      for (int c = lane * 8; c < p.d; c += kLanes * 8) {
        float v[8];
        load8(x + c, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) s = fmaf(v[j], v[j], s);
      }
#pragma unroll
    for (int o = kLanes / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (!on) continue;
    const float inv = 1.f / sqrtf(s * p.inv_q + p.eps);
    T* dst = is_q ? static_cast<T*>(p.q_out) + (t * p.heads + h) * p.d
                  : static_cast<T*>(p.k_cache) + ((page * p.hkv + h - p.heads) * p.page + off) * p.d;
    for (int c = lane * 8; c < p.d; c += kLanes * 8) {
      float v[8];
      turned8(p, x, is_q ? p.wq : p.wk, inv, cs, c, v);
      store8(dst + c, v);
    }
  }
  if (slot < 0) return;
  const int vvec = p.dv >> 3;
  for (int i = threadIdx.x; i < p.hkv * vvec; i += blockDim.x) {
    const int h = i / vvec, c = (i - h * vvec) * 8;
    float v[8];
    load8(row + p.v_off + h * p.dv + c, v);
    store8(static_cast<T*>(p.v_cache) + ((page * p.hkv + h) * p.page + off) * p.dv + c, v);
  }
}

}  // namespace b200

using namespace b200;

// out [tokens][pairs] (cos, sin) of position * (hi + lo)
B200_API int b200_rope_table(const int* positions, const float* hi, const float* lo, void* out, int tokens, int pairs, cudaStream_t stream) {
  if (tokens <= 0 || pairs <= 0) return 0;
  const long long n = static_cast<long long>(tokens) * pairs;
  const cudaError_t e = launch_pdl(rope_table_kernel, dim3(static_cast<unsigned>((n + 255) / 256)), dim3(256), 0, stream, positions, hi, lo,
                                   static_cast<float2*>(out), n, pairs);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

// See the header comment. d, dv, offsets and ld multiples of 8; q_true / k_true: how many values of q and k are the
// model's (the rest is zero padding); rot even, at most d.
B200_API int b200_qk_rope_store(const void* p, const void* wq, const void* wk, const void* table, void* q_out, void* k_cache, void* v_cache,
                                const long long* slots, int tokens, long long ld, int heads, int hkv, int d, int dv, int k_off, int v_off,
                                int page, int rot, int interleaved, int q_true, int k_true, float eps, int f32, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (ld % 8 || d % 8 || dv % 8 || k_off % 8 || v_off % 8 || rot % 2 || rot > d || page < 1 || q_true < 1 || k_true < 1) return -2;
  QkRopeParams a{p, static_cast<const __nv_bfloat16*>(wq), static_cast<const __nv_bfloat16*>(wk),
                 rot > 0 ? static_cast<const float2*>(table) : nullptr, q_out, k_cache, v_cache, slots, ld, heads, hkv, d, dv, k_off, v_off,
                 page, rot, interleaved, 1.f / q_true, 1.f / k_true, eps};
  const int vecs = (heads * d + hkv * (d + dv)) / 8;
  int threads = (vecs + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const cudaError_t e = f32 ? launch_pdl(qk_rope_store_kernel<float>, dim3(tokens), dim3(threads), 0, stream, a)
                            : launch_pdl(qk_rope_store_kernel<__nv_bfloat16>, dim3(tokens), dim3(threads), 0, stream, a);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

// See the header comment: as b200_qk_rope_store with weights [d] that all heads share and a norm per head of its d_true
// values. hkv 0: q only (wk and the caches are not used).
B200_API int b200_head_norm_store(const void* p, const void* wq, const void* wk, const void* table, void* q_out, void* k_cache, void* v_cache,
                                  const long long* slots, int tokens, long long ld, int heads, int hkv, int d, int dv, int k_off, int v_off,
                                  int page, int rot, int interleaved, int d_true, float eps, int f32, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (ld % 8 || d % 8 || dv % 8 || k_off % 8 || v_off % 8 || rot % 2 || rot > d || page < 1 || d_true < 1 || !wq || (hkv && !wk)) return -2;
  QkRopeParams a{p, static_cast<const __nv_bfloat16*>(wq), static_cast<const __nv_bfloat16*>(wk),
                 rot > 0 ? static_cast<const float2*>(table) : nullptr, q_out, k_cache, v_cache, slots, ld, heads, hkv, d, dv, k_off, v_off,
                 page, rot, interleaved, 1.f / d_true, 1.f / d_true, eps};
  const int lanes = d <= 64 ? 8 : d <= 128 ? 16 : 32;
  int threads = ((heads + hkv) * lanes + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  auto go = [&](auto kernel) { return launch_pdl(kernel, dim3(tokens), dim3(threads), 0, stream, a); };
  cudaError_t e;
  if (f32) e = lanes == 8 ? go(head_norm_store_kernel<float, 8>) : lanes == 16 ? go(head_norm_store_kernel<float, 16>) : go(head_norm_store_kernel<float, 32>);
  else e = lanes == 8 ? go(head_norm_store_kernel<__nv_bfloat16, 8>) : lanes == 16 ? go(head_norm_store_kernel<__nv_bfloat16, 16>)
                                                                            : go(head_norm_store_kernel<__nv_bfloat16, 32>);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}
