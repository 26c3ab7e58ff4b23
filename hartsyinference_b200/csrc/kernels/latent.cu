// Pieces of latent attention, with or without a rotated part, any head count and sizes.
//
// Per token the cache holds one RMS-normed latent c; per head k = W_uk c and v = W_uv c. With a rotated part the row
// goes on with one rotated key vector that all heads share, and each head's query has a part of that size. Queries come through a
// normed latent of their own. Decoding and short runs attend over the cached latents with W_uk moved to the query
// side and W_uv behind the softmax (mla.cu); long runs of a prompt expand keys and values of their context once
// (attention.cu, the contiguous form).
//
//  * latent_prep    both latents' RMS norms and the key's rotation in one launch: the query latent to a dense
//                   matrix, the key / value latent and the rotated key straight into their page.
//  * latent_gather  cached rows of sequences (from a given token on), in order, for the expansion.
//  * head_linear    one small product per head, out[t][h] = W[h] x[t][h], optionally times sigmoid(gate): the
//                   query-side W_uk (its first column block also turns the query's rotated part and moves it behind
//                   the product), and W_uv with the output gate in its epilogue. Warp-level mma.sync: with at
//                   most a few hundred rows per head it is bound by reading the weights.
#include "mixer_common.cuh"
#include "mma_sync.cuh"

namespace b200 {

struct LatentPrepParams {
  const void* p;             // [T][ld]: query latent at q_off, key / value latent at kv_off
  const __nv_bfloat16 *wq, *wkv;
  void* cq;                  // [T][q_cols]
  void* cache;               // [slots][kv_cols]
  const long long* slots;    // [T], < 0: not stored
  long long ld;
  int tokens, q_off, q_dim, q_cols, kv_off, kv_dim, kv_cols;    // dims: true sizes; cols: laid out (rest zero)
  float eps;
  const float2* table;       // [T][rot / 2] (cos, sin) of the key's rotated part behind the latent, pairs (2i, 2i + 1)
  int rot, rot_cols;         // its true and laid-out size (0: none); cache rows are kv_cols + rot_cols long
};

// One warp per (token, latent): even warps the query's, odd warps the cached one. 256 threads.
template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentPrepParams p) {
  pdl_wait();
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long t = blockIdx.x * 4 + (warp >> 1);
  if (t >= p.tokens) return;
  const bool kv = warp & 1;
  const int dim = kv ? p.kv_dim : p.q_dim, cols = kv ? p.kv_cols : p.q_cols;
  T* dst = static_cast<T*>(p.cq) + t * cols;
  if (kv) {
    const long long slot = p.slots[t];
    if (slot < 0) return;
    dst = static_cast<T*>(p.cache) + slot * (cols + p.rot_cols);
    const T* rs = static_cast<const T*>(p.p) + t * p.ld + p.kv_off + cols;
    for (int i = lane; i < p.rot_cols / 2; i += 32) {
      float a = 0.f, b = 0.f;
      if (2 * i < p.rot) {
        const float2 cs = p.table[t * (p.rot / 2) + i];
        const float u = ld1(rs + 2 * i), v = ld1(rs + 2 * i + 1);
        a = u * cs.x - v * cs.y;
        b = v * cs.x + u * cs.y;
      }
      dst[cols + 2 * i] = static_cast<T>(a);
      dst[cols + 2 * i + 1] = static_cast<T>(b);
    }
  }
  const T* src = static_cast<const T*>(p.p) + t * p.ld + (kv ? p.kv_off : p.q_off);
  const __nv_bfloat16* w = kv ? p.wkv : p.wq;
  float v[4][8];                             // up to 1024 values stay in registers
  float q = 0.f;
  for (int i = 0, c = lane * 8; c < cols; ++i, c += 256) {
    float u[8];
    load8(src + c, u);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c + j >= dim) u[j] = 0.f;
      q = fmaf(u[j], u[j], q);
    }
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (k == i)
#pragma unroll
        for (int j = 0; j < 8; ++j) v[k][j] = u[j];
  }
  const float inv = 1.f / sqrtf(warp_sum(q) / dim + p.eps);
  for (int i = 0, c = lane * 8; c < cols; ++i, c += 256) {
    float u[8], wv[8];
    if (i >= 4) load8(src + c, u);
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (k == i)
#pragma unroll
        for (int j = 0; j < 8; ++j) u[j] = v[k][j];
    load8(w + c, wv);
#pragma unroll
    for (int j = 0; j < 8; ++j) u[j] = c + j < dim ? u[j] * inv * wv[j] : 0.f;
    store8(dst + c, u);
  }
}

// out[off[s] + i] = cache row of token starts[s] + i of sequence seq_ids[s]; 16 bytes per thread. grid (blocks, seqs)
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint8_t* __restrict__ cache, uint8_t* __restrict__ out,
                                                            const int* __restrict__ block_table, const int* __restrict__ seq_ids,
                                                            const int* __restrict__ offsets, const int* __restrict__ starts, int vecs,
                                                            int page, int max_pages) {
  pdl_wait();
  pdl_trigger();
  const int s = blockIdx.y, off = offsets[s], n = offsets[s + 1] - off, first = starts ? starts[s] : 0;
  const int* table = block_table + static_cast<long long>(seq_ids[s]) * max_pages;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < static_cast<long long>(n) * vecs;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const int t = static_cast<int>(i / vecs), c = static_cast<int>(i % vecs);
    const int at = first + t;
    const long long row = static_cast<long long>(table[at / page]) * page + at % page;
    reinterpret_cast<uint4*>(out)[(off + t) * static_cast<long long>(vecs) + c] = reinterpret_cast<const uint4*>(cache)[row * vecs + c];
  }
}

struct HeadLinearParams {
  const void* x;             // row r, head h: x + r * ldx + h * x_stride, k values
  const __nv_bfloat16* w;    // [heads * n][k]
  void* out;                 // row r, head h: out + r * ldo + h * o_stride, n values
  const void* gate;          // row r, head h: gate + r * ldg + h * o_stride (head_gate: one value at h), or null
  const int* in_rows;        // row of x for product row i, or null
  const int* out_rows;       // row of out and gate for product row i, or null
  long long ldx, ldo, ldg;
  int rows, n, k, x_stride, o_stride;
  // tail > 0: the tail values behind a head's k are turned by table [token][rot / 2] (cos, sin) of their row of x, pairs
  // (2i, 2i + 1), zero from rot on, and stored behind the head's n
  const float2* table;
  int rot, tail;
  int head_gate;
};

// The tail of the rows m0 .. m0 + count of one head.
template <typename T>
__device__ __forceinline__ void head_tail(const HeadLinearParams& p, int m0, int count, int head) {
  const int pairs = p.tail / 2;
  for (int u = threadIdx.x; u < count * pairs; u += blockDim.x) {
    const int i = m0 + u / pairs, j = u % pairs;
    if (i >= p.rows) break;
    const long long src = p.in_rows ? p.in_rows[i] : i, dst = p.out_rows ? p.out_rows[i] : i;
    float a = 0.f, b = 0.f;
    if (2 * j < p.rot) {
      const float2 cs = p.table[src * (p.rot / 2) + j];
      const T* x = static_cast<const T*>(p.x) + src * p.ldx + static_cast<long long>(head) * p.x_stride + p.k + 2 * j;
      const float s = ld1(x), t = ld1(x + 1);
      a = s * cs.x - t * cs.y;
      b = t * cs.x + s * cs.y;
    }
    T* o = static_cast<T*>(p.out) + dst * p.ldo + static_cast<long long>(head) * p.o_stride + p.n + 2 * j;
    o[0] = static_cast<T>(a);
    o[1] = static_cast<T>(b);
  }
}

constexpr int kHlM = 64, kHlK = 64, kHlStages = 3;

// grid (ceil(rows / 64), ceil(n / kN), heads), 128 threads: warp (wm, wn) has 32 rows x kN / 2 columns
template <int kN>
__global__ void __launch_bounds__(128) head_linear_kernel(const HeadLinearParams p) {
  extern __shared__ __align__(128) uint8_t smraw[];
  pdl_wait();
  pdl_trigger();
  constexpr int kStage = (kHlM + kN) * kHlK * 2, kNt = kN / 16;
  const uint32_t base = smem_u32(smraw);
  const int m0 = blockIdx.x * kHlM, n0 = blockIdx.y * kN, head = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wm = warp & 1, wn = warp >> 1;
  const auto* x = static_cast<const __nv_bfloat16*>(p.x) + head * p.x_stride;
  const __nv_bfloat16* w = p.w + static_cast<long long>(head) * p.n * p.k;
  const int nk = (p.k + kHlK - 1) / kHlK;
  auto load = [&](int kb, int st) {
    if (kb < nk)
      for (int i = threadIdx.x; i < (kHlM + kN) * 8; i += 128) {
        const int r = i >> 3, c = i & 7, col = kb * kHlK + c * 8;
        const __nv_bfloat16* src = w;
        bool ok = col < p.k;
        if (r < kHlM) {
          ok = ok && m0 + r < p.rows;
          if (ok) src = x + (p.in_rows ? p.in_rows[m0 + r] : m0 + r) * p.ldx + col;
        } else {
          ok = ok && n0 + r - kHlM < p.n;
          if (ok) src = w + static_cast<long long>(n0 + r - kHlM) * p.k + col;
        }
        cp_async_16(base + st * kStage + r * (kHlK * 2) + ((c ^ (r & 7)) << 4), src, ok);
      }
    cp_async_commit();
  };
  float acc[2][kNt][4];
#pragma unroll
  for (int a = 0; a < 2; ++a)
#pragma unroll
    for (int i = 0; i < kNt; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[a][i][j] = 0.f;
  for (int i = 0; i < kHlStages - 1; ++i) load(i, i);
  for (int kb = 0; kb < nk; ++kb) {
    cp_async_wait<kHlStages - 2>();
    __syncthreads();
    load(kb + kHlStages - 1, (kb + kHlStages - 1) % kHlStages);
    const uint32_t st = base + kb % kHlStages * kStage;
#pragma unroll
    for (int kk = 0; kk < kHlK / 16; ++kk) {
      uint32_t a[2][4];
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const int ar = wm * 32 + m * 16 + (lane & 15), ac = kk * 2 + (lane >> 4);
        ldmatrix_x4(st + ar * (kHlK * 2) + ((ac ^ (ar & 7)) << 4), a[m][0], a[m][1], a[m][2], a[m][3]);
      }
#pragma unroll
      for (int g = 0; g < kNt / 2; ++g) {
        const int mi = lane >> 3;
        const int br = kHlM + wn * (kN / 2) + g * 16 + (lane & 7) + 8 * (mi >> 1), bc = kk * 2 + (mi & 1);
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(st + br * (kHlK * 2) + ((bc ^ (br & 7)) << 4), b0, b1, b2, b3);
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          mma_bf16_16816(acc[m][g * 2], a[m], b0, b1);
          mma_bf16_16816(acc[m][g * 2 + 1], a[m], b2, b3);
        }
      }
    }
  }
  cp_async_wait<0>();
  if (p.tail && blockIdx.y == 0) head_tail<__nv_bfloat16>(p, m0, kHlM, head);
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int i = m0 + wm * 32 + m * 16 + (lane >> 2) + 8 * r;
      if (i >= p.rows) continue;
      const long long row = p.out_rows ? p.out_rows[i] : i;
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + row * p.ldo + head * p.o_stride;
      const __nv_bfloat16* gate = nullptr;
      float scale = 1.f;
      if (p.gate && p.head_gate) scale = sigmoid_f32(ld1(static_cast<const __nv_bfloat16*>(p.gate) + row * p.ldg + head));
      else if (p.gate) gate = static_cast<const __nv_bfloat16*>(p.gate) + row * p.ldg + head * p.o_stride;
#pragma unroll
      for (int g = 0; g < kNt; ++g) {
        const int j = n0 + wn * (kN / 2) + g * 8 + (lane & 3) * 2;
        if (j >= p.n) continue;
        float u = acc[m][g][2 * r] * scale, v = acc[m][g][2 * r + 1] * scale;
        if (gate) {
          const float2 s = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + j));
          u *= sigmoid_f32(s.x);
          v *= sigmoid_f32(s.y);
        }
        *reinterpret_cast<uint32_t*>(out + j) = pack_bf16x2(u, v);
      }
    }
}

// 32-bit runs: 32 rows x 32 columns per block of 256 threads, FMA. grid as above with tiles of 32
__global__ void __launch_bounds__(256) head_linear_f32_kernel(const HeadLinearParams p) {
  __shared__ float xs[32][33], ws[32][33];
  const int m0 = blockIdx.x * 32, n0 = blockIdx.y * 32, head = blockIdx.z;
  const float* x = static_cast<const float*>(p.x) + head * p.x_stride;
  const __nv_bfloat16* w = p.w + static_cast<long long>(head) * p.n * p.k;
  const int c = threadIdx.x & 31, r0 = threadIdx.x >> 5;
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  for (int k0 = 0; k0 < p.k; k0 += 32) {
    for (int r = r0; r < 32; r += 8) {
      const int i = m0 + r, j = n0 + r, kk = k0 + c;
      xs[r][c] = i < p.rows && kk < p.k ? x[(p.in_rows ? p.in_rows[i] : i) * p.ldx + kk] : 0.f;
      ws[r][c] = j < p.n && kk < p.k ? __bfloat162float(w[static_cast<long long>(j) * p.k + kk]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int kk = 0; kk < 32; ++kk)
#pragma unroll
      for (int q = 0; q < 4; ++q) acc[q] = fmaf(xs[r0 + 8 * q][kk], ws[c][kk], acc[q]);
    __syncthreads();
  }
  if (p.tail && blockIdx.y == 0) head_tail<float>(p, m0, 32, head);
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    const int i = m0 + r0 + 8 * q, j = n0 + c;
    if (i >= p.rows || j >= p.n) continue;
    const long long row = p.out_rows ? p.out_rows[i] : i;
    float v = acc[q];
    if (p.gate) v *= sigmoid_f32(static_cast<const float*>(p.gate)[row * p.ldg + (p.head_gate ? head : head * p.o_stride + j)]);
    static_cast<float*>(p.out)[row * p.ldo + head * p.o_stride + j] = v;
  }
}

}  // namespace b200

using namespace b200;

// Offsets, columns and ld are multiples of 8; weights have `cols` entries (padded). rot > 0 (even): the rot_cols columns
// behind the key / value latent are a rotated key, turned by table [tokens][rot / 2] (cos, sin).
B200_API int b200_latent_prep(const void* x, const void* wq, const void* wkv, void* cq, void* cache, const long long* slots,
                              int tokens, long long ld, int q_off, int q_dim, int q_cols, int kv_off, int kv_dim, int kv_cols,
                              float eps, const void* table, int rot, int rot_cols, int f32, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (rot % 2 || rot > rot_cols || rot_cols % 8 || (rot && !table)) return -2;
  if (ld % 8 || q_off % 8 || kv_off % 8 || q_cols % 8 || kv_cols % 8 || q_dim > q_cols || kv_dim > kv_cols) return -2;
  LatentPrepParams p{x, static_cast<const __nv_bfloat16*>(wq), static_cast<const __nv_bfloat16*>(wkv), cq, cache, slots, ld,
                     tokens, q_off, q_dim, q_cols, kv_off, kv_dim, kv_cols, eps, static_cast<const float2*>(table), rot, rot_cols};
  const dim3 grid((tokens + 3) / 4);
  const cudaError_t e = f32 ? launch_pdl(latent_prep_kernel<float>, grid, dim3(256), 0, stream, p)
                            : launch_pdl(latent_prep_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, p);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

// Rows of row_bytes (a multiple of 16); offsets [seqs + 1] rows of out; max_len the longest sequence; starts [seqs]
// first token of each (null: 0).
B200_API int b200_latent_gather(const void* cache, void* out, const int* block_table, const int* seq_ids, const int* offsets,
                                const int* starts, int seqs, int max_len, int row_bytes, int page, int max_pages, cudaStream_t stream) {
  if (seqs <= 0 || max_len <= 0) return 0;
  if (row_bytes % 16 || seqs > 65535) return -2;
  const int vecs = row_bytes / 16;
  long long blocks = (static_cast<long long>(max_len) * vecs + 255) / 256;
  if (blocks > 1024) blocks = 1024;
  const cudaError_t e = launch_pdl(latent_gather_kernel, dim3(static_cast<unsigned>(blocks), seqs), dim3(256), 0, stream,
                                   static_cast<const uint8_t*>(cache), static_cast<uint8_t*>(out), block_table, seq_ids, offsets,
                                   starts, vecs, page, max_pages);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

// n, k, strides and row pitches multiples of 8; head_gate: one gate column per head; tail > 0: see HeadLinearParams
B200_API int b200_head_linear(const void* x, const void* w, void* out, const void* gate, const int* in_rows, const int* out_rows,
                              int rows, int heads, int n, int k, long long ldx, int x_stride, long long ldo, int o_stride,
                              long long ldg, const void* table, int rot, int tail, int head_gate, int f32, cudaStream_t stream) {
  if (rows <= 0 || heads <= 0) return 0;
  if (tail && (tail % 8 || rot % 2 || rot > tail || !table || x_stride < k + tail || o_stride < n + tail)) return -2;
  if (n % 8 || k % 8 || ldx % 8 || x_stride % 8 || ldo % 8 || o_stride % 8 || ldg % 8 || heads > 65535) return -2;
  HeadLinearParams p{x, static_cast<const __nv_bfloat16*>(w), out, gate, in_rows, out_rows, ldx, ldo, ldg, rows, n, k, x_stride, o_stride,
                     static_cast<const float2*>(table), rot, tail, head_gate};
  if (f32) {
    head_linear_f32_kernel<<<dim3((rows + 31) / 32, (n + 31) / 32, heads), 256, 0, stream>>>(p);
    return cudaGetLastError() == cudaSuccess ? 0 : -300;
  }
  const int mb = (rows + kHlM - 1) / kHlM;
  const bool narrow = static_cast<long long>(mb) * ((n + 63) / 64) * heads < 148;
  auto go = [&](auto kernel, int kn, PerDeviceOnce& once) {
    const int smem = kHlStages * (kHlM + kn) * kHlK * 2;
    if (once.first_time()) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    return launch_pdl(kernel, dim3(mb, (n + kn - 1) / kn, heads), dim3(128), smem, stream, p);
  };
  static PerDeviceOnce once[2];
  const cudaError_t e = narrow ? go(head_linear_kernel<32>, 32, once[0]) : go(head_linear_kernel<64>, 64, once[1]);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}
