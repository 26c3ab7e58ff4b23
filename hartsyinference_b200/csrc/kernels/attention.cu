// Attention over a paged or contiguous KV store, bf16 in / fp32 softmax / bf16 out.
//
//  * decode:  one query token per sequence; the G query heads that share a KV head form the rows
//             of the score tile, the four warps of a CTA split each 64-token KV tile, optional
//             split-KV across CTAs with a combine kernel (flash-decoding).
//  * prefill: 64 query tokens of one head per CTA (16 per warp), causal or full, KV read either
//             through the block table (chunked prefill with a cached prefix) or from contiguous
//             [tokens][heads][d] tensors (DiT self/cross attention).
//
// K/V pages are read straight from the page pool through the block table; nothing is gathered
// into a contiguous scratch first. This replaces the reference's per-sequence page gather plus
// scalar flash kernels (src/HartsyInference.LLM/Transformer/PagedKvCache.cs:116-169,
// src/HartsyInference.Cuda/Kernels/lm/flash_attn_f32.cu, flash_attn_f32_split.cu,
// flash_attn_v2_tf32.cu). Supported per-call options follow the reference's attention oracle
// (src/HartsyInference.Core/Backends/AttentionReference.cs): GQA, causal, sliding window,
// logit soft-cap. The extended form of both kernels (template flag kExt) adds, each optional: a bias
// by key distance from a per-head table or linear in the distance, a per-head sink score that only enters the
// denominator, values that are the keys themselves (one page plane), a sigmoid gate on the output (per value or per
// head), an output row pitch, first tokens that
// stay visible outside the window, key and value sizes up to 128 that are multiples of 8, and a row pitch
// for q; over contiguous keys also a part of the key that all heads share, with the rotation of its query
// side. There the probabilities keep 16 bits of
// mantissa in the PV product (a bf16 head and a bf16 remainder). `attn_rows_kernel` computes the same
// with plain fp32 arithmetic for models run in 32 bits and for shapes the tensor-core form leaves out.
//
// The score and PV products use warp-level mma.sync (m16n8k16, bf16): with one to sixteen query
// rows per KV head the kernel is bound by KV bandwidth, not by tensor throughput, and a 128-row
// tcgen05 tile would be mostly padding.
#include "common.cuh"
#include "mma_sync.cuh"

namespace b200 {

constexpr int kTileTokens = 64;
constexpr int kAttnThreads = 128;

struct AttnParams {
  const __nv_bfloat16* q;       // decode: [seqs][hq][d]; prefill: [total_q][hq][d]
  const __nv_bfloat16* k;       // paged: [pages][hkv][page][d]; contiguous: [total_kv][hkv][d]
  const __nv_bfloat16* v;
  __nv_bfloat16* out;           // same layout as q
  const int* block_table;       // [seqs][max_pages]
  const int* kv_lens;           // [seqs] keys visible to the last query token
  const int* cu_q;              // prefill: [seqs + 1] offsets into q (null -> one sequence)
  const int* cu_kv;             // contiguous prefill: [seqs + 1] offsets into k/v
  float* ws_o;                  // split partials [seqs][hq][splits][d]
  float* ws_ml;                 // [seqs][hq][splits][2]
  int seqs, hq, hkv, max_pages, page, page_shift, splits;
  int q_len_single, kv_len_single;   // used when cu_q / kv_lens are null
  int causal, window;           // window <= 0: unlimited
  float scale_log2;             // softmax scale * log2(e)
  float softcap;                // 0 = off; scores = cap * tanh(scores / cap) (pre-scale units)
  float scale;                  // plain softmax scale (needed with softcap)
  // decode, head dim 128, split path: the combine kernel also emits the output as e4m3 with one
  // scale per head (= one 1x128 group of the following linear's input), saving a quantise kernel
  uint8_t* out_q;               // [seqs][hq * d] or null
  void* out_scale;              // fp32 [seqs][hq], or blocked UE8M0 bytes when sf_tile_rows > 0
  int sf_tile_rows;
  // extended form only
  const float* dist_bias;       // [hq][dist_len] added to the score by key distance (last entry beyond it), or null
  const float* sinks;           // [hq] score of a key without a value, or null
  const __nv_bfloat16* gate;    // [tokens][gate_ld]: out *= sigmoid(gate), or null
  long long q_ld, gate_ld;      // row pitches in elements
  int dist_len, d, shared_kv;   // d: head size as stored; shared_kv: v is k
  int dv;                       // size of values and output per head
  const int* q_lens;            // [seqs] with cu_q = [seqs] starts: the listed runs need not be adjacent; or null
  long long k_ld, v_ld;         // contiguous k, v: row pitches (head h at h * d, h * dv)
  int keep;                     // window > 0: keys before this position are visible whatever the window
  // contiguous k: columns from d_own on are the same for all heads, row pitch k2_ld (d_own = d: none). With
  // rot_table [tokens][(d - d_own) / 2] (cos, sin) those columns of q are turned on the way in, pairs (2i, 2i + 1)
  const __nv_bfloat16* k2;
  const float2* rot_table;
  long long k2_ld;
  int d_own, rot_pairs;
  const float* slopes;          // [hq] slope * distance is taken off the score, or null
  int head_gate;                // gate [tokens][gate_ld] holds one column per head
  long long out_ld;             // output row pitch (head h at h * dv)
  float cap_in, cap_out;        // softcap: cap_out * tanh(score / softcap), exp(2 score / softcap) = 2^(cap_in * q.k)
};
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kDistSmem = 4096;   // longest distance table that prefill blocks keep in shared memory

__device__ __forceinline__ float exp2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Scores of one warp tile in the extended form, in place (log2 units): scale, cap, distance bias, mask.
// kMask: some key of the tile may be masked for some row. The bias table is read at fixed offsets from one
// pointer per row while the tile's distances stay inside it, and only once when they all lie past its end.
template <int NT, bool kMask>
__device__ __forceinline__ void ext_scores(float (&s)[NT][4], int key0, const int (&row_limit)[2], const int (&row_start)[2],
                                           const AttnParams& p, const float* const* row_bias, const float* row_slope) {
  int mode = -1;
  float far[2] = {0.f, 0.f};
  const float* at[2] = {nullptr, nullptr};
  if (p.dist_bias) {
    const int d0 = row_limit[0] - 1 - key0, d1 = row_limit[1] - 1 - key0;       // distances of the first key
    const int lo = min(d0, d1) - (NT * 8 - 7), hi = max(d0, d1);
    mode = __all_sync(0xffffffffu, lo >= p.dist_len - 1) ? 2 : __all_sync(0xffffffffu, lo >= 0 && hi < p.dist_len) ? 1 : 0;
    if (mode == 2) {
      far[0] = row_bias[0][p.dist_len - 1];
      far[1] = row_bias[1][p.dist_len - 1];
    }
    if (mode == 1) {
      at[0] = row_bias[0] + d0;
      at[1] = row_bias[1] + d1;
    }
  }
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (p.softcap > 0.f) {
        const float e = exp2_approx(fminf(s[nt][j] * p.cap_in, 126.f));
        s[nt][j] = p.cap_out - __fdividef(2.f * p.cap_out, e + 1.f);
      } else {
        s[nt][j] *= p.scale_log2;
      }
    }
  if (mode == 1) {
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[nt][j] = fmaf(at[j >> 1][-(nt * 8 + (j & 1))], kLog2e, s[nt][j]);
  } else if (mode == 2) {
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[nt][j] = fmaf(far[j >> 1], kLog2e, s[nt][j]);
  } else if (mode == 0) {
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int r = j >> 1;
        const int dist = min(max(row_limit[r] - 1 - (key0 + nt * 8 + (j & 1)), 0), p.dist_len - 1);
        s[nt][j] = fmaf(row_bias[r][dist], kLog2e, s[nt][j]);
      }
  }
  if (p.slopes) {
    const float back[2] = {static_cast<float>(key0 + 1 - row_limit[0]), static_cast<float>(key0 + 1 - row_limit[1])};   // minus the distance
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[nt][j] = fmaf(row_slope[j >> 1], back[j >> 1] + (nt * 8 + (j & 1)), s[nt][j]);
  }
  if (kMask) {
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int key = key0 + nt * 8 + (j & 1);
        if (key >= row_limit[j >> 1] || (key < row_start[j >> 1] && key >= p.keep)) s[nt][j] = -INFINITY;
      }
  }
}

// Tiles that a window leaves: [0, kept) of the first tokens, then [tile0, n). They are walked as one range that starts
// at tile0 - kept; tile_at gives the tile of a step.
__device__ __forceinline__ int kept_tiles(const AttnParams& p, int tile0) {
  return min((p.keep + kTileTokens - 1) / kTileTokens, tile0);
}
__device__ __forceinline__ int tile_at(int step, int tile0, int kept) { return step < tile0 ? step - (tile0 - kept) : step; }

// Shared-memory tile: [64 tokens][D] bf16, row pitch D * 2 bytes, 16-byte chunks XOR-swizzled with
// (token & 7) so that ldmatrix rows of consecutive tokens hit different banks.
template <int D>
__device__ __forceinline__ uint32_t tile_off(int token, int chunk) {
  return static_cast<uint32_t>(token * (D * 2) + ((chunk ^ (token & 7)) << 4));
}

// Loads one 64-token K or V tile through the block table. The tile's page ids were staged in
// shared memory (`pg`, 64 / page entries) an iteration earlier, so no cp.async waits on a
// dependent global load of the table; page sizes are powers of two (8..64), so token -> (page,
// offset) is a shift and a mask.
template <int D, bool kExt = false>
__device__ __forceinline__ void load_tile_paged(uint32_t smem_base, const __nv_bfloat16* pool,
                                                const int* pg, int kv_head, int hkv, int page_shift,
                                                int tok0, int kv_len, int d = D) {
  constexpr int kChunks = D / 8;
  const int page_mask = (1 << page_shift) - 1;
  for (int i = threadIdx.x; i < kTileTokens * kChunks; i += kAttnThreads) {
    const int t = i / kChunks, c = i % kChunks;
    const bool valid = tok0 + t < kv_len && (!kExt || c * 8 < d);
    const __nv_bfloat16* src = pool;
    if (valid) {
      const long long pgi = pg[t >> page_shift];
      src = pool + (((pgi * hkv + kv_head) << page_shift) + (t & page_mask)) * (kExt ? d : D) + c * 8;
    }
    cp_async_16(smem_base + tile_off<D>(t, c), src, valid);
  }
}
// Stages the page ids of step `step` (tile `tile`) into ring slot (step & 7). Tiles start on page boundaries
// because 64 is a multiple of every supported page size.
__device__ __forceinline__ void stage_pages(int (*ring)[8], const int* table, int step, int n_steps, int tile,
                                            int page_shift, int kv_len) {
  const int per_tile = kTileTokens >> page_shift;
  if (step < n_steps && threadIdx.x < per_tile) {
    const int first = (tile * kTileTokens) >> page_shift;
    const int idx = first + threadIdx.x;
    const int last_page = (kv_len - 1) >> page_shift;
    ring[step & 7][threadIdx.x] = idx <= last_page ? table[idx] : 0;
  }
}
template <int D, bool kExt = false>
__device__ __forceinline__ void load_tile_linear(uint32_t smem_base, const __nv_bfloat16* base,
                                                 long long row_stride, int tok0, int kv_len, int d = D,
                                                 const __nv_bfloat16* base2 = nullptr, long long stride2 = 0, int d_own = D) {
  constexpr int kChunks = D / 8;
  for (int i = threadIdx.x; i < kTileTokens * kChunks; i += kAttnThreads) {
    const int t = i / kChunks, c = i % kChunks;
    const int tok = tok0 + t;
    const bool valid = tok < kv_len && (!kExt || c * 8 < d);
    const __nv_bfloat16* src = valid ? base + tok * row_stride + c * 8 : base;
    if (kExt && valid && c * 8 >= d_own) src = base2 + tok * stride2 + (c * 8 - d_own);
    cp_async_16(smem_base + tile_off<D>(t, c), src, valid);
  }
}

// Per-warp flash-attention state for 16 query rows: thread (g = lane / 4, t = lane % 4) owns rows g
// and g + 8.
template <int D>
struct WarpState {
  float o[D / 8][4];
  float m[2], l[2];
  __device__ __forceinline__ void init() {
#pragma unroll
    for (int i = 0; i < D / 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) o[i][j] = 0.f;
    m[0] = m[1] = -INFINITY;
    l[0] = l[1] = 0.f;
  }
};

// Processes NG groups of 16 tokens starting at tile-local token `t_begin` for this warp.
//   qf: Q fragments [D/16][4]; row_limit[r]: first masked key position for the thread's row r
//   (keys >= limit are masked), row_start[r]: first visible key (sliding window).
//   Extended form: row_bias[r] is the row's distance-bias table (the distance of a key is counted back
//   from row_limit[r] - 1), row_slope[r] its slope times log2(e).
template <int D, int NG, bool kExt = false, int DV = D>
__device__ __forceinline__ void warp_tile(WarpState<DV>& st, const uint32_t (&qf)[D / 16][4],
                                          uint32_t k_smem, uint32_t v_smem, int t_begin,
                                          int tok0, const int (&row_limit)[2],
                                          const int (&row_start)[2], const AttnParams& p,
                                          const float* const* row_bias = nullptr, const float* row_slope = nullptr) {
  const int lane = threadIdx.x & 31;
  const int tq = lane & 3;
  float s[NG * 2][4];
#pragma unroll
  for (int i = 0; i < NG * 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
  // S = Q K^T
#pragma unroll
  for (int kk = 0; kk < D / 16; ++kk) {
#pragma unroll
    for (int gi = 0; gi < NG; ++gi) {
      const int mi = lane >> 3;
      const int token = t_begin + gi * 16 + (lane & 7) + 8 * (mi >> 1);
      const int chunk = kk * 2 + (mi & 1);
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4(k_smem + tile_off<D>(token, chunk), b0, b1, b2, b3);
      mma_bf16_16816(s[gi * 2], qf[kk], b0, b1);
      mma_bf16_16816(s[gi * 2 + 1], qf[kk], b2, b3);
    }
  }
  // scale, soft-cap, mask; running max
  float mx[2] = {-INFINITY, -INFINITY};
  if (kExt) {
    const int first = tok0 + t_begin, last = first + NG * 16 - 1;
    const bool open = last < min(row_limit[0], row_limit[1]) && (first >= max(row_start[0], row_start[1]) || last < p.keep);
    if (__all_sync(0xffffffffu, open)) ext_scores<NG * 2, false>(s, first + tq * 2, row_limit, row_start, p, row_bias, row_slope);
    else ext_scores<NG * 2, true>(s, first + tq * 2, row_limit, row_start, p, row_bias, row_slope);
  }
#pragma unroll
  for (int nt = 0; nt < NG * 2; ++nt) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = j >> 1;
      const int key = tok0 + t_begin + nt * 8 + tq * 2 + (j & 1);
      float x = s[nt][j];
      if (kExt) {
        mx[r] = fmaxf(mx[r], x);
        continue;
      }
      if (p.softcap > 0.f) x = p.softcap * tanhf(x * p.scale / p.softcap) * (p.scale_log2 / p.scale);
      else x *= p.scale_log2;
      if (key >= row_limit[r] || key < row_start[r]) x = -INFINITY;
      s[nt][j] = x;
      mx[r] = fmaxf(mx[r], x);
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
    mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
  }
  float alpha[2], msafe[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const float mnew = fmaxf(st.m[r], mx[r]);
    msafe[r] = mnew == -INFINITY ? 0.f : mnew;
    alpha[r] = st.m[r] == -INFINITY ? 0.f : exp2f(st.m[r] - msafe[r]);
    st.m[r] = mnew;
  }
  float rs[2] = {0.f, 0.f};
  uint32_t pf[NG][4], pl[kExt ? NG : 1][4];
#pragma unroll
  for (int nt = 0; nt < NG * 2; ++nt) {
    float e[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      e[j] = kExt ? exp2_approx(s[nt][j] - msafe[j >> 1]) : exp2f(s[nt][j] - msafe[j >> 1]);
      rs[j >> 1] += e[j];
    }
    // A fragment of P for the 16-token group nt / 2: (a0, a1) from the even n-tile, (a2, a3)
    // from the odd one
    pf[nt >> 1][(nt & 1) * 2 + 0] = pack_bf16x2(e[0], e[1]);
    pf[nt >> 1][(nt & 1) * 2 + 1] = pack_bf16x2(e[2], e[3]);
    if (kExt) {
#pragma unroll
      for (int j = 0; j < 4; ++j) e[j] -= __bfloat162float(__float2bfloat16(e[j]));
      pl[kExt ? nt >> 1 : 0][(nt & 1) * 2 + 0] = pack_bf16x2(e[0], e[1]);
      pl[kExt ? nt >> 1 : 0][(nt & 1) * 2 + 1] = pack_bf16x2(e[2], e[3]);
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    rs[r] += __shfl_xor_sync(0xffffffffu, rs[r], 1);
    rs[r] += __shfl_xor_sync(0xffffffffu, rs[r], 2);
    st.l[r] = st.l[r] * alpha[r] + rs[r];
  }
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) {
    st.o[i][0] *= alpha[0];
    st.o[i][1] *= alpha[0];
    st.o[i][2] *= alpha[1];
    st.o[i][3] *= alpha[1];
  }
  // O += P V
#pragma unroll
  for (int gi = 0; gi < NG; ++gi) {
#pragma unroll
    for (int np = 0; np < DV / 16; ++np) {
      const int mi = lane >> 3;
      const int token = t_begin + gi * 16 + (lane & 7) + 8 * (mi & 1);
      const int chunk = np * 2 + (mi >> 1);
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4_trans(v_smem + tile_off<DV>(token, chunk), b0, b1, b2, b3);
      mma_bf16_16816(st.o[np * 2], pf[gi], b0, b1);
      mma_bf16_16816(st.o[np * 2 + 1], pf[gi], b2, b3);
      if (kExt) {
        mma_bf16_16816(st.o[np * 2], pl[kExt ? gi : 0], b0, b1);
        mma_bf16_16816(st.o[np * 2 + 1], pl[kExt ? gi : 0], b2, b3);
      }
    }
  }
}

__device__ __forceinline__ float gate_of(const AttnParams& p, long long token, int head, int c) {
  return p.gate ? 1.f / (1.f + __expf(-__bfloat162float(p.gate[token * p.gate_ld + (p.head_gate ? head : head * p.dv + c)]))) : 1.f;
}

// ------------------------------------------------------------------------------------------
// decode
// ------------------------------------------------------------------------------------------
template <int D, int kStages, bool kExt = false>
__global__ void __launch_bounds__(kAttnThreads)
attn_decode_kernel(const AttnParams p) {
  pdl_wait();
  pdl_trigger();
  constexpr int kTileBytes = kTileTokens * D * 2;
  extern __shared__ __align__(128) uint8_t smem[];
  const int stage_bytes = kExt && p.shared_kv ? kTileBytes : 2 * kTileBytes;
  const int seq = blockIdx.x, kvh = blockIdx.y, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, tq = lane & 3;
  const int G = p.hq / p.hkv;
  const int kv_len = p.kv_lens[seq];
  const int n_tiles = (kv_len + kTileTokens - 1) / kTileTokens;
  const int start_key = p.window > 0 ? max(0, kv_len - p.window) : 0;
  const int tile0 = start_key / kTileTokens;                    // tiles before the window are not read
  const int kept = kExt ? kept_tiles(p, tile0) : 0;             // except those of the kept first tokens
  const int tiles_per_split = (n_tiles - tile0 + kept + p.splits - 1) / p.splits;
  const int tile_begin = tile0 - kept + split * tiles_per_split;
  const int tile_end = min(n_tiles, tile_begin + tiles_per_split);
  const int* table = p.block_table + static_cast<long long>(seq) * p.max_pages;
  const uint32_t smem_base = smem_u32(smem);

  // Q fragments: row = query head within the group (rows >= G are zero)
  uint32_t qf[D / 16][4];
  {
    const int d = kExt ? p.d : D;
    const __nv_bfloat16* qb = kExt ? p.q + seq * p.q_ld + kvh * G * d : p.q + (static_cast<long long>(seq) * p.hq + kvh * G) * D;
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      const int c0 = kk * 16 + tq * 2;
      if (kExt) {
        qf[kk][0] = g < G && c0 < d ? *reinterpret_cast<const uint32_t*>(qb + g * d + c0) : 0u;
        qf[kk][1] = g + 8 < G && c0 < d ? *reinterpret_cast<const uint32_t*>(qb + (g + 8) * d + c0) : 0u;
        qf[kk][2] = g < G && c0 + 8 < d ? *reinterpret_cast<const uint32_t*>(qb + g * d + c0 + 8) : 0u;
        qf[kk][3] = g + 8 < G && c0 + 8 < d ? *reinterpret_cast<const uint32_t*>(qb + (g + 8) * d + c0 + 8) : 0u;
        continue;
      }
      qf[kk][0] = g < G ? *reinterpret_cast<const uint32_t*>(qb + g * D + c0) : 0u;
      qf[kk][1] = g + 8 < G ? *reinterpret_cast<const uint32_t*>(qb + (g + 8) * D + c0) : 0u;
      qf[kk][2] = g < G ? *reinterpret_cast<const uint32_t*>(qb + g * D + c0 + 8) : 0u;
      qf[kk][3] = g + 8 < G ? *reinterpret_cast<const uint32_t*>(qb + (g + 8) * D + c0 + 8) : 0u;
    }
  }
  WarpState<D> st;
  st.init();
  const int lim[2] = {kv_len, kv_len};
  const int start[2] = {start_key, start_key};
  const float* row_bias[2] = {nullptr, nullptr};
  float row_slope[2] = {0.f, 0.f};
  if (kExt) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int head = kvh * G + min(g + 8 * r, G - 1);
      if (p.slopes) row_slope[r] = p.slopes[head] * kLog2e;
      if (p.dist_bias) row_bias[r] = p.dist_bias + static_cast<long long>(head) * p.dist_len;
      if (p.sinks && split == 0 && warp == 0) {       // the sink enters the running sums once
        st.m[r] = p.sinks[head] * kLog2e;
        st.l[r] = 1.f;
      }
    }
  }

  __shared__ int pg_ring[8][8];
  auto tile_of = [&](int step) { return kExt ? tile_at(step, tile0, kept) : step; };
  auto stage = [&](int step) { stage_pages(pg_ring, table, step, tile_end, tile_of(step), p.page_shift, kv_len); };
  auto issue = [&](int step, int slot) {
    if (step < tile_end) {
      const uint32_t kb = smem_base + slot * stage_bytes;
      const int* pages = pg_ring[step & 7];
      const int tok0 = tile_of(step) * kTileTokens;
      if (kExt) {
        load_tile_paged<D, true>(kb, p.k, pages, kvh, p.hkv, p.page_shift, tok0, kv_len, p.d);
        if (!p.shared_kv) load_tile_paged<D, true>(kb + kTileBytes, p.v, pages, kvh, p.hkv, p.page_shift, tok0, kv_len, p.dv);
        cp_async_commit();
        return;
      }
      load_tile_paged<D>(kb, p.k, pages, kvh, p.hkv, p.page_shift, tok0, kv_len);
      load_tile_paged<D>(kb + kTileBytes, p.v, pages, kvh, p.hkv, p.page_shift, tok0, kv_len);
    }
    cp_async_commit();
  };
  stage(tile_begin);
  stage(tile_begin + 1);
  stage(tile_begin + 2);
  if (kStages > 3) stage(tile_begin + 3);
  __syncthreads();
#pragma unroll
  for (int i = 0; i < kStages - 1; ++i) issue(tile_begin + i, i);
  int slot = 0;
  for (int step = tile_begin; step < tile_end; ++step) {
    // these page ids are read by issue() in a later iteration, after two barriers
    stage(step + (kStages > 3 ? kStages : 3));
    issue(step + kStages - 1, (slot + kStages - 1) % kStages);
    cp_async_wait<kStages - 1>();
    __syncthreads();
    const uint32_t kb = smem_base + slot * stage_bytes;
    warp_tile<D, 1, kExt>(st, qf, kb, kExt && p.shared_kv ? kb : kb + kTileBytes, warp * 16, tile_of(step) * kTileTokens, lim, start,
                          p, row_bias, row_slope);
    __syncthreads();
    slot = (slot + 1) % kStages;
  }
  cp_async_wait<0>();
  __syncthreads();

  // merge the four warps' partial states through shared memory
  float* so = reinterpret_cast<float*>(smem);                    // [4][16][D]
  float* sml = so + 4 * 16 * D;                                  // [4][16][2]
#pragma unroll
  for (int i = 0; i < D / 8; ++i) {
    const int c = i * 8 + tq * 2;
    so[(warp * 16 + g) * D + c] = st.o[i][0];
    so[(warp * 16 + g) * D + c + 1] = st.o[i][1];
    so[(warp * 16 + g + 8) * D + c] = st.o[i][2];
    so[(warp * 16 + g + 8) * D + c + 1] = st.o[i][3];
  }
  if (tq == 0) {
    sml[(warp * 16 + g) * 2] = st.m[0];
    sml[(warp * 16 + g) * 2 + 1] = st.l[0];
    sml[(warp * 16 + g + 8) * 2] = st.m[1];
    sml[(warp * 16 + g + 8) * 2 + 1] = st.l[1];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < G * D; i += kAttnThreads) {
    const int r = i / D, c = i % D;
    float mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, sml[(w * 16 + r) * 2]);
    float acc = 0.f, ll = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float mw = sml[(w * 16 + r) * 2];
      const float f = mw == -INFINITY ? 0.f : exp2f(mw - mm);
      acc += so[(w * 16 + r) * D + c] * f;
      ll += sml[(w * 16 + r) * 2 + 1] * f;
    }
    const int head = kvh * G + r;
    if (kExt && p.splits == 1) {
      if (c < p.dv)
        p.out[seq * p.out_ld + head * p.dv + c] = __float2bfloat16((ll > 0.f ? acc / ll : 0.f) * gate_of(p, seq, head, c));
    } else if (p.splits == 1) {
      p.out[(static_cast<long long>(seq) * p.hq + head) * D + c] =
          __float2bfloat16(ll > 0.f ? acc / ll : 0.f);
    } else {
      const long long base = (static_cast<long long>(seq) * p.hq + head) * p.splits + split;
      p.ws_o[base * D + c] = acc;
      if (c == 0) {
        p.ws_ml[base * 2] = mm;
        p.ws_ml[base * 2 + 1] = ll;
      }
    }
  }
}

template <int D, bool kExt = false>
__global__ void attn_combine_kernel(const AttnParams p) {
  pdl_wait();
  pdl_trigger();
  const int seq = blockIdx.x, head = blockIdx.y;
  const long long base = (static_cast<long long>(seq) * p.hq + head) * p.splits;
  float mm = -INFINITY;
  for (int s = 0; s < p.splits; ++s) mm = fmaxf(mm, p.ws_ml[(base + s) * 2]);
  for (int c = threadIdx.x; c < D; c += blockDim.x) {
    float acc = 0.f, ll = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float ms = p.ws_ml[(base + s) * 2];
      const float f = ms == -INFINITY ? 0.f : exp2f(ms - mm);
      acc += p.ws_o[(base + s) * D + c] * f;
      ll += p.ws_ml[(base + s) * 2 + 1] * f;
    }
    if (kExt) {
      if (c < p.dv)
        p.out[seq * p.out_ld + head * p.dv + c] = __float2bfloat16((ll > 0.f ? acc / ll : 0.f) * gate_of(p, seq, head, c));
      continue;
    }
    const __nv_bfloat16 o = __float2bfloat16(ll > 0.f ? acc / ll : 0.f);
    if (p.out) p.out[(static_cast<long long>(seq) * p.hq + head) * D + c] = o;
    if (D == 128 && p.out_q) {
      // blockDim == D: every thread holds one value of the head; the head is one quantisation group
      __shared__ float wmax[4];
      const float v = __bfloat162float(o);
      float amax = warp_max(fabsf(v));
      if ((threadIdx.x & 31) == 0) wmax[threadIdx.x >> 5] = amax;
      __syncthreads();
      amax = fmaxf(fmaxf(wmax[0], wmax[1]), fmaxf(wmax[2], wmax[3]));
      float sc = fmaxf(amax, 1e-12f) / 448.f, inv = 1.f / sc;
      uint32_t eb = 127;
      if (p.sf_tile_rows > 0) {
        // UE8M0: the smallest power of two >= amax / 448
        const uint32_t bits = __float_as_uint(amax / 448.f);
        int e = static_cast<int>(bits >> 23) - 127 + ((bits & 0x7fffffu) != 0 ? 1 : 0);
        e = max(-126, min(126, e));
        eb = static_cast<uint32_t>(e + 127);
        inv = __uint_as_float(static_cast<uint32_t>(127 - e) << 23);
      }
      p.out_q[(static_cast<long long>(seq) * p.hq + head) * D + c] =
          static_cast<uint8_t>(__nv_cvt_float_to_fp8(v * inv, __NV_SATFINITE, __NV_E4M3));
      if (c == 0) {
        if (p.sf_tile_rows > 0) {
          // blocked layout: row tiles of sf_tile_rows, K groups of four 128-wide blocks, row r of a
          // tile at word (r % 32) * 4 + r / 32, K block kb at byte kb % 4
          const int kgroups = (p.hq * D + 511) >> 9;
          const int tile = seq / p.sf_tile_rows, r = seq - tile * p.sf_tile_rows;
          const long long blk = static_cast<long long>(tile) * kgroups + (head >> 2);
          static_cast<uint8_t*>(p.out_scale)[(blk * 128 + (r & 31) * 4 + (r >> 5)) * 4 + (head & 3)] =
              static_cast<uint8_t>(eb);
        } else {
          static_cast<float*>(p.out_scale)[static_cast<long long>(seq) * p.hq + head] = sc;
        }
      }
    }
  }
}

// ------------------------------------------------------------------------------------------
// prefill / full attention
// ------------------------------------------------------------------------------------------
// DV: width of the value tiles (D but for keys of 192, which come with values of at most 128)
template <int D, bool kPaged, bool kExt = false, int DV = D>
__global__ void __launch_bounds__(kAttnThreads)
attn_prefill_kernel(const AttnParams p) {
  constexpr int kStages = 2;
  constexpr int kTileBytes = kTileTokens * D * 2;
  extern __shared__ __align__(128) uint8_t smem[];
  const int qt = blockIdx.x, head = blockIdx.y, seq = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, tq = lane & 3;
  const int G = p.hq / p.hkv;
  const int kvh = head / G;
  const int q_off = p.cu_q ? p.cu_q[seq] : 0;
  const int q_len = kExt && p.q_lens ? p.q_lens[seq] : p.cu_q ? p.cu_q[seq + 1] - q_off : p.q_len_single;
  const int kv_len = p.kv_lens ? p.kv_lens[seq] : p.kv_len_single;
  if (qt * 64 >= q_len) return;
  const int stage_bytes = kExt && p.shared_kv ? kTileBytes : kTileBytes + kTileTokens * DV * 2;
  const int ctx = kv_len - q_len;   // keys that precede the first query token
  const uint32_t smem_base = smem_u32(smem);

  const int row0 = qt * 64 + warp * 16 + g;   // this thread's rows: row0, row0 + 8
  uint32_t qf[D / 16][4];
  {
    const int d = kExt ? p.d : D;
    const __nv_bfloat16* qb = kExt ? p.q + q_off * p.q_ld + head * d : p.q + (static_cast<long long>(q_off) * p.hq + head) * D;
    const long long rs = kExt ? p.q_ld : static_cast<long long>(p.hq) * D;
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      const int c0 = kk * 16 + tq * 2;
      if (kExt) {
        qf[kk][0] = row0 < q_len && c0 < d ? *reinterpret_cast<const uint32_t*>(qb + row0 * rs + c0) : 0u;
        qf[kk][1] = row0 + 8 < q_len && c0 < d ? *reinterpret_cast<const uint32_t*>(qb + (row0 + 8) * rs + c0) : 0u;
        qf[kk][2] = row0 < q_len && c0 + 8 < d ? *reinterpret_cast<const uint32_t*>(qb + row0 * rs + c0 + 8) : 0u;
        qf[kk][3] = row0 + 8 < q_len && c0 + 8 < d ? *reinterpret_cast<const uint32_t*>(qb + (row0 + 8) * rs + c0 + 8) : 0u;
        continue;
      }
      qf[kk][0] = row0 < q_len ? *reinterpret_cast<const uint32_t*>(qb + row0 * rs + c0) : 0u;
      qf[kk][1] = row0 + 8 < q_len ? *reinterpret_cast<const uint32_t*>(qb + (row0 + 8) * rs + c0) : 0u;
      qf[kk][2] = row0 < q_len ? *reinterpret_cast<const uint32_t*>(qb + row0 * rs + c0 + 8) : 0u;
      qf[kk][3] = row0 + 8 < q_len ? *reinterpret_cast<const uint32_t*>(qb + (row0 + 8) * rs + c0 + 8) : 0u;
    }
  }
  if (kExt && !kPaged && p.rot_table) {
    // a thread's values come in pairs of neighbours: turn those of the shared part
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int pair = (kk * 16 + tq * 2 + 8 * (i >> 1) - p.d_own) >> 1, row = row0 + 8 * (i & 1);
        if (pair >= 0 && pair < p.rot_pairs && row < q_len) {
          const float2 cs = p.rot_table[static_cast<long long>(q_off + row) * p.rot_pairs + pair];
          const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&qf[kk][i]));
          qf[kk][i] = pack_bf16x2(v.x * cs.x - v.y * cs.y, v.y * cs.x + v.x * cs.y);
        }
      }
  }
  WarpState<DV> st;
  st.init();
  int lim[2], start[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int pos = ctx + row0 + 8 * r;   // absolute position of the query row
    lim[r] = p.causal ? min(kv_len, pos + 1) : kv_len;
    start[r] = p.window > 0 ? max(0, pos + 1 - p.window) : 0;
  }
  const float* row_bias[2] = {nullptr, nullptr};
  float row_slope[2] = {0.f, 0.f};
  if (kExt) {
    if (p.slopes) row_slope[0] = row_slope[1] = p.slopes[head] * kLog2e;
    if (p.dist_bias) {
      row_bias[0] = row_bias[1] = p.dist_bias + static_cast<long long>(head) * p.dist_len;
      if (p.dist_len <= kDistSmem) {
        float* tab = reinterpret_cast<float*>(smem + 2 * stage_bytes);
        for (int i = threadIdx.x; i < p.dist_len; i += kAttnThreads) tab[i] = row_bias[0][i];
        row_bias[0] = row_bias[1] = tab;                // visible after the first barrier of the tile loop
      }
    }
    if (p.sinks) {
      st.m[0] = st.m[1] = p.sinks[head] * kLog2e;
      st.l[0] = st.l[1] = 1.f;
    }
  }
  // keys needed by this CTA: up to the last row's position when causal
  const int last_pos = ctx + min(q_len, qt * 64 + 64) - 1;
  const int kv_needed = p.causal ? min(kv_len, last_pos + 1) : kv_len;
  const int n_tiles = (kv_needed + kTileTokens - 1) / kTileTokens;
  int tile0 = 0;
  if (p.window > 0) tile0 = max(0, ctx + qt * 64 + 1 - p.window) / kTileTokens;
  const int kept = kExt ? kept_tiles(p, tile0) : 0;

  const int* table = kPaged ? p.block_table + static_cast<long long>(seq) * p.max_pages : nullptr;
  const int kv_off = (!kPaged && p.cu_kv) ? p.cu_kv[seq] : 0;
  const long long kv_rs = static_cast<long long>(p.hkv) * D;
  const __nv_bfloat16* kbase = kPaged ? p.k : kExt ? p.k + kv_off * p.k_ld + kvh * p.d_own : p.k + (static_cast<long long>(kv_off) * p.hkv + kvh) * D;
  const __nv_bfloat16* k2base = kExt && !kPaged && p.k2 ? p.k2 + kv_off * p.k2_ld : nullptr;
  const __nv_bfloat16* vbase = kPaged ? p.v : kExt ? p.v + kv_off * p.v_ld + kvh * p.dv : p.v + (static_cast<long long>(kv_off) * p.hkv + kvh) * D;

  __shared__ int pg_ring[8][8];
  auto tile_of = [&](int step) { return kExt ? tile_at(step, tile0, kept) : step; };
  auto stage = [&](int step) { stage_pages(pg_ring, table, step, n_tiles, tile_of(step), p.page_shift, kv_needed); };
  auto issue = [&](int step, int slot) {
    if (step < n_tiles) {
      const uint32_t kb = smem_base + slot * stage_bytes;
      const int* pages = pg_ring[step & 7];
      const int tok0 = tile_of(step) * kTileTokens;
      if (kExt && !kPaged) {
        load_tile_linear<D, true>(kb, kbase, p.k_ld, tok0, kv_needed, p.d, k2base, p.k2_ld, p.d_own);
        load_tile_linear<DV, true>(kb + kTileBytes, vbase, p.v_ld, tok0, kv_needed, p.dv);
      } else if (kExt) {
        load_tile_paged<D, true>(kb, p.k, pages, kvh, p.hkv, p.page_shift, tok0, kv_needed, p.d);
        if (!p.shared_kv) load_tile_paged<D, true>(kb + kTileBytes, p.v, pages, kvh, p.hkv, p.page_shift, tok0, kv_needed, p.dv);
      } else if (kPaged) {
        load_tile_paged<D>(kb, p.k, pages, kvh, p.hkv, p.page_shift, tok0, kv_needed);
        load_tile_paged<D>(kb + kTileBytes, p.v, pages, kvh, p.hkv, p.page_shift, tok0, kv_needed);
      } else {
        load_tile_linear<D>(kb, kbase, kv_rs, tok0, kv_needed);
        load_tile_linear<D>(kb + kTileBytes, vbase, kv_rs, tok0, kv_needed);
      }
    }
    cp_async_commit();
  };
  const int first = tile0 - kept;
  if (kPaged) {
    stage(first);
    stage(first + 1);
    __syncthreads();
  }
  issue(first, 0);
  int slot = 0;
  for (int step = first; step < n_tiles; ++step) {
    if (kPaged) stage(step + 2);
    issue(step + 1, slot ^ 1);
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t kb = smem_base + slot * stage_bytes;
    // a warp whose rows all lie before this tile (causal) still runs: masked scores cost nothing
    // in correctness and keep the barrier pattern uniform
    warp_tile<D, 4, kExt, DV>(st, qf, kb, kExt && p.shared_kv ? kb : kb + kTileBytes, 0, tile_of(step) * kTileTokens, lim, start, p,
                          row_bias, row_slope);
    __syncthreads();
    slot ^= 1;
  }
  cp_async_wait<0>();
  static_assert(kStages == 2, "double buffered");

  __nv_bfloat16* ob = p.out + (static_cast<long long>(q_off) * p.hq + head) * D;
  const long long rs = static_cast<long long>(p.hq) * D;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = row0 + 8 * r;
    if (row < q_len) {
      float inv = st.l[r] > 0.f ? 1.f / st.l[r] : 0.f;
      if (kExt && p.head_gate) inv *= gate_of(p, q_off + row, head, 0);
#pragma unroll
      for (int i = 0; i < DV / 8; ++i) {
        const int c = i * 8 + tq * 2;
        if (kExt) {
          float a = st.o[i][2 * r] * inv, b = st.o[i][2 * r + 1] * inv;
          if (c >= p.dv) continue;
          if (!p.head_gate) {
            a *= gate_of(p, q_off + row, head, c);
            b *= gate_of(p, q_off + row, head, c + 1);
          }
          *reinterpret_cast<uint32_t*>(p.out + (q_off + row) * p.out_ld + head * p.dv + c) = pack_bf16x2(a, b);
          continue;
        }
        *reinterpret_cast<uint32_t*>(ob + row * rs + c) =
            pack_bf16x2(st.o[i][2 * r] * inv, st.o[i][2 * r + 1] * inv);
      }
    }
  }
}

// ------------------------------------------------------------------------------------------
// plain form: one warp per (token, head), 32 keys at a time, fp32 arithmetic throughout
// ------------------------------------------------------------------------------------------
struct AttnRowsParams {
  const void *q, *k, *v, *gate;
  void* out;
  const int *block_table, *kv_lens, *cu_q;
  const float *dist_bias, *sinks;
  long long q_ld, gate_ld;
  int tokens, seqs, hq, hkv, d, page, max_pages, window, dist_len;
  float scale, softcap;
  int keep, dv, v_row;         // kept first tokens; value size, and values per row of the value pages
  const float* slopes;         // as in AttnParams
  int head_gate;
  long long out_ld;
};
constexpr int kRowsMaxD = 1024, kRowsMaxV = 512;   // query-key and value size

__device__ __forceinline__ float as_f32(float v) { return v; }
__device__ __forceinline__ float as_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T>
__global__ void __launch_bounds__(128) attn_rows_kernel(const AttnRowsParams p) {
  pdl_wait();
  pdl_trigger();
  __shared__ float qs[4][kRowsMaxD];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * 4 + warp, head = blockIdx.y;
  if (t >= p.tokens) return;
  int seq = t, first = t, q_len = 1;
  if (p.cu_q) {
    int lo = 0, hi = p.seqs - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.cu_q[mid] <= t) lo = mid; else hi = mid - 1;
    }
    seq = lo;
    first = p.cu_q[seq];
    q_len = p.cu_q[seq + 1] - first;
  }
  const int pos = p.kv_lens[seq] - q_len + (t - first);      // -1 for an empty sequence: no keys
  const int begin = p.window > 0 ? max(0, pos + 1 - p.window) : 0;
  const int kept = min(p.keep, begin), keys = kept + pos + 1 - begin;       // [0, kept) and [begin, pos]
  const int kvh = head / (p.hq / p.hkv);
  const int* table = p.block_table + static_cast<long long>(seq) * p.max_pages;
  const T* q = static_cast<const T*>(p.q) + t * p.q_ld + head * p.d;
  for (int c = lane; c < p.d; c += 32) qs[warp][c] = as_f32(q[c]);
  __syncwarp();
  float m = p.sinks ? p.sinks[head] : -INFINITY, l = p.sinks ? 1.f : 0.f;
  float o[kRowsMaxV / 32];
#pragma unroll
  for (int i = 0; i < kRowsMaxV / 32; ++i) o[i] = 0.f;
  for (int j0 = 0; j0 < keys; j0 += 32) {
    const int j = j0 + lane < kept ? j0 + lane : begin + j0 + lane - kept;
    long long at = 0;
    float s = -INFINITY;
    if (j0 + lane < keys) {
      at = (static_cast<long long>(table[j / p.page]) * p.hkv + kvh) * p.page + j % p.page;
      const T* kr = static_cast<const T*>(p.k) + at * p.d;
      float a = 0.f;
      for (int c = 0; c < p.d; ++c) a += qs[warp][c] * as_f32(kr[c]);
      s = a * p.scale;
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      if (p.dist_bias) s += p.dist_bias[static_cast<long long>(head) * p.dist_len + min(pos - j, p.dist_len - 1)];
      if (p.slopes) s -= p.slopes[head] * static_cast<float>(pos - j);
    }
    const float mn = fmaxf(m, warp_max(s));
    const float f = m == -INFINITY ? 0.f : expf(m - mn);
    const float e = s == -INFINITY ? 0.f : expf(s - mn);
    l = l * f + warp_sum(e);
    m = mn;
#pragma unroll
    for (int i = 0; i < kRowsMaxV / 32; ++i) o[i] *= f;
    const int n = min(32, keys - j0);
    for (int jj = 0; jj < n; ++jj) {
      const float w = __shfl_sync(0xffffffffu, e, jj);
      const T* vr = static_cast<const T*>(p.v) + __shfl_sync(0xffffffffu, at, jj) * p.v_row;
#pragma unroll
      for (int i = 0; i < kRowsMaxV / 32; ++i)
        if (lane + i * 32 < p.dv) o[i] += w * as_f32(vr[lane + i * 32]);
    }
  }
  T* out = static_cast<T*>(p.out) + t * p.out_ld + head * p.dv;
  const T* gate = p.gate ? static_cast<const T*>(p.gate) + t * p.gate_ld + (p.head_gate ? head : head * p.dv) : nullptr;
#pragma unroll
  for (int i = 0; i < kRowsMaxV / 32; ++i) {
    const int c = lane + i * 32;
    if (c < p.dv) {
      float y = l > 0.f ? o[i] / l : 0.f;
      if (gate) y *= 1.f / (1.f + expf(-as_f32(gate[p.head_gate ? 0 : c])));
      out[c] = static_cast<T>(y);
    }
  }
}

// Rows of keys (and values) into their pages: [tokens][ld] -> [pages][hkv][page][row], 16 bytes per thread
__global__ void kv_store_kernel(const uint8_t* __restrict__ k, const uint8_t* __restrict__ v, uint8_t* __restrict__ kc,
                                uint8_t* __restrict__ vc, const long long* __restrict__ slots, int tokens, int hkv,
                                int row_vecs, int page, long long ld_bytes) {
  pdl_wait();
  pdl_trigger();
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= static_cast<long long>(tokens) * hkv * row_vecs) return;
  const int c = static_cast<int>(i % row_vecs), h = static_cast<int>(i / row_vecs % hkv);
  const long long t = i / row_vecs / hkv, slot = slots[t];
  if (slot < 0) return;
  const long long src = t * ld_bytes + (static_cast<long long>(h) * row_vecs + c) * 16;
  const long long dst = (((slot / page) * hkv + h) * page + slot % page) * row_vecs + c;
  reinterpret_cast<uint4*>(kc)[dst] = *reinterpret_cast<const uint4*>(k + src);
  if (v) reinterpret_cast<uint4*>(vc)[dst] = *reinterpret_cast<const uint4*>(v + src);
}

}  // namespace b200

using namespace b200;

B200_API long long b200_attn_decode_workspace_bytes(int seqs, int hq, int d, int splits) {
  return splits > 1 ? static_cast<long long>(seqs) * hq * splits * (d + 2) * 4 : 0;
}

static int g_decode_stages = 2;

// Number of KV splits for a decode batch, from a wave model fitted to B200 timings: the grid runs
// in waves of (148 SMs x resident CTAs) and a CTA costs its tiles plus about four tiles' worth of
// prologue and merge, so the estimate is waves x (ceil(tiles / splits) + 4); ties go to fewer
// splits (less partial traffic and a cheaper combine). Measured with the two-tile ring, 64-token
// tiles, 2304-token contexts (CTAs before splitting: best splits, time): 16: 12, 13.5 us;
// 64: 6, 24.9 us; 128: 3, 40.4 us; 256: 3 or 1, 76-78 us; 512: 2, 132 us (8192 tokens: 4, 388 us;
// 512 tokens: 1, 41 us); 1024: 1, 238 us.
B200_API int b200_attn_decode_pick_splits(int seqs, int hkv, int max_kv_len) {
  const int ctas = seqs * hkv > 0 ? seqs * hkv : 1;
  const int tiles = (max_kv_len + kTileTokens - 1) / kTileTokens;
  const int slots = 148 * (g_decode_stages == 2 ? 3 : 2);
  int best = 1;
  long long best_cost = -1;
  for (int sp = 1; sp <= 16 && sp <= tiles; ++sp) {
    const long long waves = (static_cast<long long>(ctas) * sp + slots - 1) / slots;
    const long long cost = waves * ((tiles + sp - 1) / sp + 4);
    if (best_cost < 0 || cost < best_cost) { best_cost = cost; best = sp; }
  }
  return best;
}


// Depth of the decode kernel's K/V staging ring: 3 (two CTAs per SM at head dim 128) or 2 (three).
B200_API void b200_attn_set_decode_stages(int stages) { g_decode_stages = stages == 2 ? 2 : 3; }

B200_API int b200_attn_decode(const void* q, const void* k_cache, const void* v_cache, void* out,
                              const int* block_table, const int* kv_lens, int seqs, int hq, int hkv,
                              int d, int page, int max_pages, int splits, void* workspace,
                              float scale, float softcap, int window, void* out_q, void* out_scale,
                              int sf_tile_rows, cudaStream_t stream) {
  if (seqs <= 0) return 0;
  if (out_q != nullptr && (d != 128 || splits <= 1 || out_scale == nullptr)) return -6;   // combine kernel only
  if (d != 64 && d != 128) return -2;
  if (hq % hkv != 0 || hq / hkv > 16) return -3;
  if (splits > 1 && !workspace) return -5;
  AttnParams p{};
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.k = static_cast<const __nv_bfloat16*>(k_cache);
  p.v = static_cast<const __nv_bfloat16*>(v_cache);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.block_table = block_table;
  p.kv_lens = kv_lens;
  p.seqs = seqs; p.hq = hq; p.hkv = hkv; p.max_pages = max_pages; p.page = page;
  p.page_shift = page == 8 ? 3 : page == 16 ? 4 : page == 32 ? 5 : page == 64 ? 6 : -1;
  if (p.page_shift < 0) return -4;
  p.splits = splits < 1 ? 1 : splits;
  p.window = window;
  p.scale = scale;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.softcap = softcap;
  p.out_q = static_cast<uint8_t*>(out_q);
  p.out_scale = out_scale;
  p.sf_tile_rows = sf_tile_rows;
  if (p.splits > 1) {
    p.ws_o = static_cast<float*>(workspace);
    p.ws_ml = p.ws_o + static_cast<long long>(seqs) * hq * p.splits * d;
  }
  dim3 grid(seqs, hkv, p.splits);
  // staging ring depth: 3 tiles (two CTAs per SM at d = 128) or 2 tiles (three CTAs per SM)
  const int stages = g_decode_stages == 2 ? 2 : 3;
  const int smem = stages * 2 * kTileTokens * d * 2;
  static PerDeviceOnce attr_set[2][2];
  PerDeviceOnce& once = attr_set[d == 128 ? 1 : 0][stages - 2];
  auto launch = [&](auto kernel) {
    if (once.first_time()) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    launch_pdl(kernel, grid, dim3(kAttnThreads), smem, stream, p);
  };
  if (d == 128) {
    if (stages == 2) launch(attn_decode_kernel<128, 2>); else launch(attn_decode_kernel<128, 3>);
  } else {
    if (stages == 2) launch(attn_decode_kernel<64, 2>); else launch(attn_decode_kernel<64, 3>);
  }
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return -static_cast<int>(e) - 300;
  if (p.splits > 1) {
    dim3 cg(seqs, hq);
    if (d == 128) launch_pdl(attn_combine_kernel<128>, cg, dim3(128), 0, stream, p);
    else launch_pdl(attn_combine_kernel<64>, cg, dim3(64), 0, stream, p);
    e = cudaGetLastError();
    if (e != cudaSuccess) return -static_cast<int>(e) - 400;
  }
  return 0;
}

// Prefill / full attention. paged != 0: k, v are page pools read through block_table and kv_lens;
// else k, v are contiguous [tokens][hkv][d] with optional cu_kv offsets.
B200_API int b200_attn_prefill(const void* q, const void* k, const void* v, void* out,
                               const int* block_table, const int* kv_lens, const int* cu_q,
                               const int* cu_kv, int seqs, int max_q_len, int q_len_single,
                               int kv_len_single, int hq, int hkv, int d, int page, int max_pages,
                               int paged, int causal, int window, float scale, float softcap,
                               cudaStream_t stream) {
  if (seqs <= 0 || max_q_len <= 0) return 0;
  if (d != 64 && d != 128) return -2;
  if (hq % hkv != 0) return -3;
  AttnParams p{};
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.k = static_cast<const __nv_bfloat16*>(k);
  p.v = static_cast<const __nv_bfloat16*>(v);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.block_table = block_table;
  p.kv_lens = kv_lens;
  p.cu_q = cu_q;
  p.cu_kv = cu_kv;
  p.seqs = seqs; p.hq = hq; p.hkv = hkv; p.max_pages = max_pages; p.page = page; p.splits = 1;
  p.page_shift = page == 8 ? 3 : page == 16 ? 4 : page == 32 ? 5 : page == 64 ? 6 : -1;
  if (paged && p.page_shift < 0) return -4;
  p.q_len_single = q_len_single; p.kv_len_single = kv_len_single;
  p.causal = causal; p.window = window;
  p.scale = scale;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.softcap = softcap;
  dim3 grid((max_q_len + 63) / 64, hq, seqs);
  const int smem = 2 * 2 * kTileTokens * d * 2;
#define LAUNCH_PREFILL(DD, PG)                                                                   \
  do {                                                                                           \
    static PerDeviceOnce once;                                                                   \
    if (once.first_time())                                                                       \
      cudaFuncSetAttribute(attn_prefill_kernel<DD, PG>,                                          \
                           cudaFuncAttributeMaxDynamicSharedMemorySize, smem);                   \
    attn_prefill_kernel<DD, PG><<<grid, kAttnThreads, smem, stream>>>(p);                        \
  } while (0)
  if (d == 128) {
    if (paged) LAUNCH_PREFILL(128, true); else LAUNCH_PREFILL(128, false);
  } else {
    if (paged) LAUNCH_PREFILL(64, true); else LAUNCH_PREFILL(64, false);
  }
#undef LAUNCH_PREFILL
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

// Extended attention over pages (see the header comment). cu_q null: one query token per sequence.
// q [tokens][q_ld] (head h at h * d), out [tokens][out_ld] (head h at h * dv). v_cache null: the values are the keys (with exact, their
// first dv columns). window > 0: the last `window` keys and the first keep_first of the sequence.
// exact != 0: plain fp32 kernel, tensors are fp32 when f32 is set and bf16 otherwise; exact == 0: the
// tensor-core kernels (bf16, d, dv <= 128, at most 16 query heads per key head at decode; returns -6 for
// what they do not take). splits / workspace: decode only, as in b200_attn_decode (with the head size
// rounded up to 64 or 128). slopes: a bias linear in the distance; head_gate: one gate column per head.
B200_API int b200_attn_biased(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_table,
                              const int* kv_lens, const int* cu_q, int tokens, int seqs, int max_q_len, int hq, int hkv, int d,
                              int dv, int page, int max_pages, int splits, void* workspace, float scale, float softcap, int window, int keep_first,
                              const float* dist_bias, int dist_len, const float* sinks, const void* gate, long long gate_ld,
                              long long q_ld, int exact, int f32, const float* slopes, int head_gate, long long out_ld,
                              cudaStream_t stream) {
  if (tokens <= 0 || seqs <= 0) return 0;
  if (d % 8 || d < 8 || d > kRowsMaxD || dv % 8 || dv < 8 || dv > kRowsMaxV || (!v_cache && dv > d) || keep_first < 0 || hq % hkv || q_ld % 8 || (gate && gate_ld % 8) || (dist_bias && dist_len < 1) || out_ld < static_cast<long long>(hq) * dv || out_ld % 8) return -2;
  if (f32 && !exact) return -6;
  if (window <= 0) keep_first = 0;
  if (exact) {
    AttnRowsParams p{q, k_cache, v_cache ? v_cache : k_cache, gate, out, block_table, kv_lens, cu_q, dist_bias, sinks,
                     q_ld, gate_ld, tokens, seqs, hq, hkv, d, page, max_pages, window, dist_len, scale, softcap,
                     keep_first, dv, v_cache ? dv : d, slopes, head_gate, out_ld};
    const dim3 grid((tokens + 3) / 4, hq);
    const cudaError_t e = f32 ? launch_pdl(attn_rows_kernel<float>, grid, dim3(128), 0, stream, p)
                              : launch_pdl(attn_rows_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, p);
    return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
  }
  if (d > 128 || dv > 128 || (!v_cache && dv != d) || (!cu_q && hq / hkv > 16)) return -6;
  AttnParams p{};
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.k = static_cast<const __nv_bfloat16*>(k_cache);
  p.v = static_cast<const __nv_bfloat16*>(v_cache ? v_cache : k_cache);
  p.shared_kv = v_cache == nullptr;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.block_table = block_table;
  p.kv_lens = kv_lens;
  p.cu_q = cu_q;
  p.seqs = seqs; p.hq = hq; p.hkv = hkv; p.max_pages = max_pages; p.page = page;
  p.page_shift = page == 8 ? 3 : page == 16 ? 4 : page == 32 ? 5 : page == 64 ? 6 : -1;
  if (p.page_shift < 0) return -4;
  p.causal = 1;
  p.window = window;
  p.scale = scale;
  p.scale_log2 = scale * kLog2e;
  p.softcap = softcap;
  if (softcap > 0.f) {
    p.cap_in = 2.f * kLog2e * scale / softcap;
    p.cap_out = softcap * kLog2e;
  }
  p.dist_bias = dist_bias; p.dist_len = dist_len; p.sinks = sinks; p.slopes = slopes; p.head_gate = head_gate; p.out_ld = out_ld;
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.gate_ld = gate_ld; p.q_ld = q_ld; p.d = p.d_own = d; p.dv = dv; p.keep = keep_first;
  p.splits = cu_q || splits < 1 ? 1 : splits;
  const int dd = d <= 64 && dv <= 64 ? 64 : 128;
  if (cu_q) {
    if (max_q_len <= 0) return 0;
    const dim3 grid((max_q_len + 63) / 64, hq, seqs);
    const int smem = 2 * (p.shared_kv ? 1 : 2) * kTileTokens * dd * 2 + (dist_bias && dist_len <= kDistSmem ? dist_len * 4 : 0);
    const int most = 2 * 2 * kTileTokens * dd * 2 + kDistSmem * 4;
    static PerDeviceOnce once[2];
    if (dd == 128) {
      if (once[1].first_time()) cudaFuncSetAttribute(attn_prefill_kernel<128, true, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
      attn_prefill_kernel<128, true, true><<<grid, kAttnThreads, smem, stream>>>(p);
    } else {
      if (once[0].first_time()) cudaFuncSetAttribute(attn_prefill_kernel<64, true, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
      attn_prefill_kernel<64, true, true><<<grid, kAttnThreads, smem, stream>>>(p);
    }
    const cudaError_t e = cudaGetLastError();
    return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
  }
  if (p.splits > 1) {
    if (!workspace) return -5;
    p.ws_o = static_cast<float*>(workspace);
    p.ws_ml = p.ws_o + static_cast<long long>(seqs) * hq * p.splits * dd;
  }
  const dim3 grid(seqs, hkv, p.splits);
  // the ring (two tiles of keys and values, or four tiles of keys that are also the values) doubles as the
  // buffer of the four warps' partial results
  const int ring = 4 * kTileTokens * dd * 2, merge = 4 * 16 * (dd + 2) * 4;
  const int smem = ring > merge ? ring : merge;
  auto go = [&](auto kernel, PerDeviceOnce& once) {
    if (once.first_time()) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    return launch_pdl(kernel, grid, dim3(kAttnThreads), smem, stream, p);
  };
  static PerDeviceOnce once[4];
  cudaError_t e;
  if (dd == 128) e = p.shared_kv ? go(attn_decode_kernel<128, 4, true>, once[0]) : go(attn_decode_kernel<128, 2, true>, once[1]);
  else e = p.shared_kv ? go(attn_decode_kernel<64, 4, true>, once[2]) : go(attn_decode_kernel<64, 2, true>, once[3]);
  if (e != cudaSuccess) return -static_cast<int>(e) - 300;
  if (p.splits > 1) {
    if (dd == 128) e = launch_pdl(attn_combine_kernel<128, true>, dim3(seqs, hq), dim3(128), 0, stream, p);
    else e = launch_pdl(attn_combine_kernel<64, true>, dim3(seqs, hq), dim3(64), 0, stream, p);
    if (e != cudaSuccess) return -static_cast<int>(e) - 400;
  }
  return 0;
}

// Causal attention of the runs q_start[s] .. + q_lens[s] of q over contiguous keys and values of their whole
// contexts (rows kv_start[s] .. + kv_lens[s] of k and v; the last key belongs to the run's last query; window > 0: the
// last `window` keys of every query). q, out and gate are indexed by token: q [tokens][q_ld] (head h at h * d), out
// [tokens][out_ld] (head h at h * dv); head_gate: one gate column per head. d <= 192, dv <= 128, multiples of 8. The keys' columns from d_own on are rows of k2 for every head
// (d_own = d: none); with rot_table [tokens][rot_pairs] (cos, sin) those columns of q are turned.
B200_API int b200_attn_runs(const void* q, const void* k, const void* v, void* out, const void* gate, const int* q_start,
                            const int* q_lens, const int* kv_start, const int* kv_lens, int seqs, int max_q_len, int hq, int hkv,
                            int d, int dv, long long q_ld, long long k_ld, long long v_ld, long long gate_ld, float scale, int window,
                            const void* k2, int d_own, long long k2_ld, const void* rot_table, int rot_pairs, const float* sinks, int head_gate,
                            long long out_ld, cudaStream_t stream) {
  if (seqs <= 0 || max_q_len <= 0) return 0;
  if (d % 8 || dv % 8 || d < 8 || dv < 8 || d > 192 || dv > 128 || hq % hkv || q_ld % 8 || k_ld % 8 || v_ld % 8 || gate_ld % 8 ||
      seqs > 65535)
    return -2;
  if (out_ld % 8 || out_ld < static_cast<long long>(hq) * dv) return -2;
  if (d_own % 8 || d_own > d || k2_ld % 8 || (d_own < d && !k2) || (rot_table && 2 * rot_pairs > d - d_own)) return -2;
  AttnParams p{};
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.k = static_cast<const __nv_bfloat16*>(k);
  p.v = static_cast<const __nv_bfloat16*>(v);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.cu_q = q_start; p.q_lens = q_lens; p.cu_kv = kv_start; p.kv_lens = kv_lens;
  p.seqs = seqs; p.hq = hq; p.hkv = hkv; p.splits = 1;
  p.causal = 1;
  p.window = window;
  p.scale = scale;
  p.scale_log2 = scale * kLog2e;
  p.d = d; p.dv = dv; p.q_ld = q_ld; p.k_ld = k_ld; p.v_ld = v_ld; p.gate_ld = gate_ld;
  p.k2 = static_cast<const __nv_bfloat16*>(k2); p.d_own = d_own; p.k2_ld = k2_ld;
  p.rot_table = static_cast<const float2*>(rot_table); p.rot_pairs = rot_pairs;
  p.sinks = sinks; p.head_gate = head_gate; p.out_ld = out_ld;
  const dim3 grid((max_q_len + 63) / 64, hq, seqs);
  auto go = [&](auto kernel, int dd, PerDeviceOnce& once) {
    const int smem = 2 * kTileTokens * (dd + (dd > 128 ? 128 : dd)) * 2;
    if (once.first_time()) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    kernel<<<grid, kAttnThreads, smem, stream>>>(p);
  };
  static PerDeviceOnce once[3];
  if (d > 128) go(attn_prefill_kernel<192, false, true, 128>, 192, once[2]);
  else if (d > 64 || dv > 64) go(attn_prefill_kernel<128, false, true>, 128, once[1]);
  else go(attn_prefill_kernel<64, false, true>, 64, once[0]);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

// k (and v, may be null) rows [tokens][ld] with hkv heads of d values of esz bytes -> page pools
B200_API int b200_kv_store(const void* k, const void* v, void* k_cache, void* v_cache, const long long* slots, int tokens,
                           int hkv, int d, int page, long long ld, int esz, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (d * esz % 16 || ld * esz % 16 || ((reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15)) return -2;
  const int vecs = d * esz / 16;
  const long long total = static_cast<long long>(tokens) * hkv * vecs;
  const cudaError_t e = launch_pdl(kv_store_kernel, dim3(static_cast<unsigned>((total + 255) / 256)), dim3(256), 0, stream,
                                   static_cast<const uint8_t*>(k), static_cast<const uint8_t*>(v),
                                   static_cast<uint8_t*>(k_cache), static_cast<uint8_t*>(v_cache), slots, tokens, hkv, vecs,
                                   page, ld * esz);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}
