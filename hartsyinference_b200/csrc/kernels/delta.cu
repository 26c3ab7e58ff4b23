// Gated delta-rule mixer with one decay per head and key channel.
//
// Per head and sequence a matrix S [dk][dv] in fp32, updated by every token t:
//   S' = Diag(g_t) S_{t-1};   S_t = S' + k_t (beta_t (v_t - S'^T k_t))^T;   o_t = S_t^T q_t
//   y_t = sigmoid(gate_t) w o_t / rms(o_t)
// q, k, v come from projections through a short causal convolution and silu; q and k are made unit
// vectors; g = exp(-A softplus(z + dt_bias)); several heads can share one q / k head.
//
//  * delta_prep     one warp per (token, head slice): convolution + silu, unit norms, decay, beta.
//                   At decode it also advances the convolution state (the last taps - 1 inputs).
//  * delta_tail     convolution state after a portion of a prompt.
//  * delta_scan     portions of prompts: the columns of S are independent, so a block takes 32 of
//                   them (a thread keeps two columns of an eighth of the rows in registers) and walks
//                   over the tokens, which are staged through shared memory. The result does not
//                   depend on where a prompt is cut: the same operations run in the same order.
//  * delta_gate     the output norm and gate of a scanned portion, one warp per (token, head).
//  * delta_step     decode: one block per (sequence, head) reads the state once, applies the update,
//                   writes it back and emits the normed, gated output.
//
// State lives in slots, [slots][heads][dk][dv] fp32 and [slots][taps - 1][channels]; a sequence whose
// portion starts at position 0 starts from zeros whatever its slot held before, a negative slot is
// computed from zeros and stored nowhere (padding rows of a captured decode batch).
#include "mixer_common.cuh"

namespace b200 {

struct DeltaParams {
  const void* proj;          // [T][ldp]: q (hk * dk) | k (hk * dk) | v (h * dv) | ..., beta logits at b_off
  const void* z;             // [T][ldz]: decay logits (h * dk), then output gate logits (h * dv) at gate_off
  const float* conv_w;       // [taps][channels]
  const float* a;            // [h] decay rate exp(A_log)
  const float* dt_bias;      // [h * dk]
  void* conv_state;          // [slots][taps - 1][channels]
  float* state;              // [slots][h][dk][dv]
  const __nv_bfloat16* norm_w;   // [dv]
  const int* positions;      // [T]
  const int* cu_q;           // [seqs + 1]; null: one token per sequence
  const int* slots;          // [seqs]
  float *q, *k, *v, *g, *beta, *o;   // scratch: [T][hk * dk] x 2, [T][h * dv], [T][h * dk], [T][h], [T][h * dv]
  void* out;                 // [T][h * dv]
  long long ldp, ldz;
  int tokens, seqs, h, hk, dk, dv, taps, b_off, gate_off, dv_true;
  float q_scale, eps;
};

constexpr int kDeltaMaxDk = 256;

// grid: (ceil(T / 8), 2 hk + 2 h); 256 threads, warp w handles token 8 * blockIdx.x + w
template <typename T>
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaParams p) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= p.tokens) return;
  const T* row = static_cast<const T*>(p.proj) + static_cast<long long>(t) * p.ldp;
  int slice = blockIdx.y;
  if (slice >= 2 * p.hk + p.h) {          // decay (and beta) of one head
    const int head = slice - 2 * p.hk - p.h;
    const float a = p.a[head];
    const T* zr = static_cast<const T*>(p.z) + static_cast<long long>(t) * p.ldz + head * p.dk;
    float* gr = p.g + (static_cast<long long>(t) * p.h + head) * p.dk;
    for (int e = lane * 4; e < p.dk; e += 128) {
      float z[4], b[4], g[4];
      ld4(zr + e, z);
      ld4(p.dt_bias + head * p.dk + e, b);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float x = z[j] + b[j];
        g[j] = decay_of(a * (fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)))));
      }
      st4(gr + e, g);
    }
    if (lane == 0) p.beta[static_cast<long long>(t) * p.h + head] = sigmoid_f32(ld1(row + p.b_off + head));
    return;
  }
  const bool is_v = slice >= 2 * p.hk;
  const int d = is_v ? p.dv : p.dk;
  const int c0 = is_v ? 2 * p.hk * p.dk + (slice - 2 * p.hk) * p.dv : slice * p.dk;
  const int channels = 2 * p.hk * p.dk + p.h * p.dv;
  const int tail = p.taps - 1;
  const int seq = p.cu_q ? seq_of_token(p.cu_q, p.seqs, t) : t;
  const int first = p.cu_q ? p.cu_q[seq] : t;
  const int slot = p.slots[seq];
  const bool carried = slot >= 0 && p.positions[first] > 0;
  T* st = static_cast<T*>(p.conv_state) + static_cast<long long>(slot < 0 ? 0 : slot) * tail * channels;
  const bool shift = p.cu_q == nullptr && slot >= 0;
  float keep[kDeltaMaxDk / 128][4];
  float sq = 0.f;
  int it = 0;
  for (int e = lane * 4; e < d; e += 128, ++it) {
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int j = 0; j < p.taps; ++j) {
      const int src = t - tail + j;                  // token whose input this tap reads
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (src >= first) ld4(row + static_cast<long long>(src - t) * p.ldp + c0 + e, x);
      else if (carried) ld4(st + static_cast<long long>(tail + src - first) * channels + c0 + e, x);
      // decode: input j becomes row j - 1 of the state (row j has been read already)
      if (shift && j > 0) st4(st + static_cast<long long>(j - 1) * channels + c0 + e, x);
      float cw[4];
      ld4(p.conv_w + static_cast<long long>(j) * channels + c0 + e, cw);
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[i] += x[i] * cw[i];
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[i] = acc[i] * sigmoid_f32(acc[i]);
    if (is_v) {
      st4(p.v + static_cast<long long>(t) * p.h * p.dv + (c0 - 2 * p.hk * p.dk) + e, acc);
    } else {
#pragma unroll
      for (int n = 0; n < kDeltaMaxDk / 128; ++n)
        if (n == it)
#pragma unroll
          for (int i = 0; i < 4; ++i) keep[n][i] = acc[i];
#pragma unroll
      for (int i = 0; i < 4; ++i) sq += acc[i] * acc[i];
    }
  }
  if (is_v) return;
  sq = warp_sum(sq);
  const bool is_q = slice < p.hk;
  const float inv = (is_q ? p.q_scale : 1.f) / sqrtf(sq + 1e-6f);
  float* dst = (is_q ? p.q + static_cast<long long>(t) * p.hk * p.dk + slice * p.dk
                     : p.k + static_cast<long long>(t) * p.hk * p.dk + (slice - p.hk) * p.dk);
#pragma unroll
  for (int n = 0; n < kDeltaMaxDk / 128; ++n) {
    const int e = lane * 4 + n * 128;
    if (e < d) {
      float v[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) v[i] = keep[n][i] * inv;
      st4(dst + e, v);
    }
  }
}

// The same for four taps and q / k heads of at most 128: a warp keeps one slice of up to 128 channels for
// `run` consecutive tokens, so that the taps' weights and the previous inputs stay in registers.
// grid: (ceil(T / (8 run)), 2 hk + ceil(h dv / 128) + ceil(h dk / 128))
template <typename T>
__global__ void __launch_bounds__(256) delta_prep4_kernel(const DeltaParams p, int run) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const int t0 = (blockIdx.x * 8 + (threadIdx.x >> 5)) * run, t1 = min(t0 + run, p.tokens);
  if (t0 >= t1) return;
  const int vslices = (p.h * p.dv + 127) / 128;
  int slice = blockIdx.y;
  if (slice >= 2 * p.hk + vslices) {      // decay, and beta with the first slice
    slice -= 2 * p.hk + vslices;
    const int e = slice * 128 + lane * 4;
    const bool on = e < p.h * p.dk;
    float b[4] = {0.f, 0.f, 0.f, 0.f};
    if (on) ld4(p.dt_bias + e, b);
    const float a = on ? p.a[e / p.dk] : 0.f;
    for (int t = t0; t < t1; ++t) {
      if (on) {
        float z[4];
        ld4(static_cast<const T*>(p.z) + static_cast<long long>(t) * p.ldz + e, z);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float x = z[j] + b[j];
          z[j] = decay_of(a * (fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)))));
        }
        st4(p.g + static_cast<long long>(t) * p.h * p.dk + e, z);
      }
      if (slice == 0)
        for (int hd = lane; hd < p.h; hd += 32)
          p.beta[static_cast<long long>(t) * p.h + hd] =
              sigmoid_f32(ld1(static_cast<const T*>(p.proj) + static_cast<long long>(t) * p.ldp + p.b_off + hd));
    }
    return;
  }
  const bool is_v = slice >= 2 * p.hk;
  const int channels = 2 * p.hk * p.dk + p.h * p.dv;
  const int vbase = 2 * p.hk * p.dk;
  const int c = (is_v ? vbase + (slice - 2 * p.hk) * 128 : slice * p.dk) + lane * 4;
  const bool on = is_v ? c < channels : lane * 4 < p.dk;
  float w[4][4];
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) w[j][i] = 0.f;
  if (on)
#pragma unroll
    for (int j = 0; j < 4; ++j) ld4(p.conv_w + static_cast<long long>(j) * channels + c, w[j]);
  const T* x = static_cast<const T*>(p.proj) + c;
  int seq = p.cu_q ? seq_of_token(p.cu_q, p.seqs, t0) : t0;
  float in[4][4];                          // inputs of the four taps, oldest first
  bool fresh = true;
  int next = 0;                            // first token of the following sequence
  for (int t = t0; t < t1; ++t) {
    if (fresh || t >= next) {
      if (!fresh) ++seq;
      fresh = false;
      const int first = p.cu_q ? p.cu_q[seq] : t;
      next = p.cu_q ? p.cu_q[seq + 1] : t + 1;
      const int slot = p.slots[seq];
      const bool carried = slot >= 0 && p.positions[first] > 0;
      T* st = static_cast<T*>(p.conv_state) + static_cast<long long>(slot < 0 ? 0 : slot) * 3 * channels + c;
#pragma unroll
      for (int j = 0; j < 3; ++j) {
#pragma unroll
        for (int i = 0; i < 4; ++i) in[j][i] = 0.f;
        const int src = t - 3 + j;
        if (!on) continue;
        if (src >= first) ld4(x + static_cast<long long>(src) * p.ldp, in[j]);
        else if (carried) ld4(st + static_cast<long long>(3 + src - first) * channels, in[j]);
      }
      if (p.cu_q == nullptr && slot >= 0 && on) {       // decode: the state moves on by one token
        float now[4];
        ld4(x + static_cast<long long>(t) * p.ldp, now);
        st4(st, in[1]);
        st4(st + channels, in[2]);
        st4(st + 2 * channels, now);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) in[3][i] = 0.f;
    if (on) ld4(x + static_cast<long long>(t) * p.ldp, in[3]);
    float y[4], sq = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) acc += in[j][i] * w[j][i];
      y[i] = acc * sigmoid_f32(acc);
      sq += y[i] * y[i];
    }
    if (is_v) {
      if (on) st4(p.v + static_cast<long long>(t) * p.h * p.dv + (c - vbase), y);
    } else {
      sq = warp_sum(sq);
      const bool is_q = slice < p.hk;
      const float inv = (is_q ? p.q_scale : 1.f) / sqrtf(sq + 1e-6f);
#pragma unroll
      for (int i = 0; i < 4; ++i) y[i] *= inv;
      if (on) st4((is_q ? p.q + c : p.k + c - p.hk * p.dk) + static_cast<long long>(t) * p.hk * p.dk, y);
    }
#pragma unroll
    for (int j = 0; j < 3; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) in[j][i] = in[j + 1][i];
  }
}

// grid: (ceil(channels / 256), seqs)
template <typename T>
__global__ void __launch_bounds__(256) delta_tail_kernel(const DeltaParams p) {
  pdl_wait();
  pdl_trigger();
  const int channels = 2 * p.hk * p.dk + p.h * p.dv;
  const int c = blockIdx.x * 256 + threadIdx.x, seq = blockIdx.y;
  const int slot = p.slots[seq];
  if (c >= channels || slot < 0) return;
  const int first = p.cu_q[seq], len = p.cu_q[seq + 1] - first, tail = p.taps - 1;
  if (len <= 0) return;
  const bool carried = p.positions[first] > 0;
  T* st = static_cast<T*>(p.conv_state) + static_cast<long long>(slot) * tail * channels + c;
  const T* x = static_cast<const T*>(p.proj) + static_cast<long long>(first) * p.ldp + c;
  for (int j = 0; j < tail; ++j) {
    const int src = len - tail + j;      // row j + len of the old state when negative
    T v = static_cast<T>(0.f);
    if (src >= 0) v = x[static_cast<long long>(src) * p.ldp];
    else if (carried) v = st[static_cast<long long>(tail + src) * channels];
    st[static_cast<long long>(j) * channels] = v;
  }
}

constexpr int kScanTokens = 16;     // tokens per staging buffer
constexpr int kScanCols = 32;       // columns of S per block

// grid: (ceil(dv / 32), h, seqs), 128 threads. dk = 32 * NR. Lane: rows i * 32 + (lane % 8) * 4 + 0..3
// of columns 2 * (lane / 8), + 1 of the warp's eight.
template <int NR>
__global__ void __launch_bounds__(128) delta_scan_kernel(const DeltaParams p) {
  pdl_wait();
  pdl_trigger();
  constexpr int DK = NR * 32;
  constexpr int kTok = 3 * DK + kScanCols + 4;      // floats per staged token: k, q, g, v, beta
  extern __shared__ __align__(16) float sm[];
  const int head = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31, rg = lane & 7;
  const int col0 = blockIdx.x * kScanCols, lc = warp * 8 + (lane >> 3) * 2, col = col0 + lc;
  const int first = p.cu_q ? p.cu_q[seq] : seq;
  const int len = p.cu_q ? p.cu_q[seq + 1] - first : 1;
  if (len <= 0) return;
  const int slot = p.slots[seq];
  const bool carried = slot >= 0 && p.positions[first] > 0;
  const bool live = col < p.dv;
  const int kh = head / (p.h / p.hk);
  float* sp = p.state + (static_cast<long long>(slot < 0 ? 0 : slot) * p.h + head) * DK * p.dv + col;

  f32x2 s0[NR * 2], s1[NR * 2];       // two columns, row pairs
#pragma unroll
  for (int i = 0; i < NR; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      float2 a = make_float2(0.f, 0.f), b = a;
      if (carried && live) {
        const float* rp = sp + static_cast<long long>(i * 32 + rg * 4 + j * 2) * p.dv;
        a = *reinterpret_cast<const float2*>(rp);
        b = *reinterpret_cast<const float2*>(rp + p.dv);
      }
      s0[i * 2 + j] = pack2(a.x, b.x);
      s1[i * 2 + j] = pack2(a.y, b.y);
    }

  auto stage = [&](int t0, int buf) {
    float* base = sm + buf * kScanTokens * kTok;
    const int n = min(kScanTokens, len - t0);
    constexpr int kVec = DK / 4;
    for (int i = tid; i < n * 3 * kVec; i += 128) {
      const int tk = i / (3 * kVec), r = i - tk * (3 * kVec), which = r / kVec, c = (r - which * kVec) * 4;
      const long long t = first + t0 + tk;
      const float* src = which == 0 ? p.k + (t * p.hk + kh) * DK + c
                       : which == 1 ? p.q + (t * p.hk + kh) * DK + c : p.g + (t * p.h + head) * DK + c;
      copy_async_16(smem_u32(base + tk * kTok + which * DK + c), src, true);
    }
    for (int i = tid; i < n * (kScanCols / 4); i += 128) {
      const int tk = i / (kScanCols / 4), c = (i % (kScanCols / 4)) * 4;
      const long long t = first + t0 + tk;
      const bool ok = col0 + c < p.dv;
      copy_async_16(smem_u32(base + tk * kTok + 3 * DK + c), ok ? p.v + (t * p.h + head) * p.dv + col0 + c : p.v, ok);
    }
    if (tid < n) {
      const long long t = first + t0 + tid;
      copy_async_4(smem_u32(base + tid * kTok + 3 * DK + kScanCols), p.beta + t * p.h + head, true);
    }
  };
  auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };

  stage(0, 0);
  commit();
  int buf = 0;
  for (int t0 = 0; t0 < len; t0 += kScanTokens, buf ^= 1) {
    if (t0 + kScanTokens < len) stage(t0 + kScanTokens, buf ^ 1);
    commit();
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const int n = min(kScanTokens, len - t0);
    const float* base = sm + buf * kScanTokens * kTok;
    float* op = p.o + (static_cast<long long>(first + t0) * p.h + head) * p.dv + col;
    ulonglong2 nk[NR], ng[NR];           // the next token's k and g, read while the current one is computed
    auto fetch = [&](int tk) {
      const float* tb = base + tk * kTok;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        nk[i] = *reinterpret_cast<const ulonglong2*>(tb + i * 32 + rg * 4);
        ng[i] = *reinterpret_cast<const ulonglong2*>(tb + 2 * DK + i * 32 + rg * 4);
      }
    };
    fetch(0);
    for (int tq = 0; tq < n; tq += 4) {
      float part[8];                       // reads of four tokens x two columns, this lane's rows
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        part[2 * j] = part[2 * j + 1] = 0.f;
        if (tq + j >= n) continue;
        const float* tb = base + (tq + j) * kTok;
        f32x2 kk[NR * 2];
        f32x2 a0 = 0, a1 = 0, b0 = 0, b1 = 0;
        const float2 v = *reinterpret_cast<const float2*>(tb + 3 * DK + lc);
        const float beta = tb[3 * DK + kScanCols];
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          kk[i * 2] = nk[i].x;
          kk[i * 2 + 1] = nk[i].y;
          s0[i * 2] = mul2(s0[i * 2], ng[i].x);
          s1[i * 2] = mul2(s1[i * 2], ng[i].x);
          s0[i * 2 + 1] = mul2(s0[i * 2 + 1], ng[i].y);
          s1[i * 2 + 1] = mul2(s1[i * 2 + 1], ng[i].y);
          a0 = fma2(s0[i * 2], nk[i].x, a0);
          a1 = fma2(s1[i * 2], nk[i].x, a1);
          b0 = fma2(s0[i * 2 + 1], nk[i].y, b0);
          b1 = fma2(s1[i * 2 + 1], nk[i].y, b1);
        }
        ulonglong2 qv[NR];
#pragma unroll
        for (int i = 0; i < NR; ++i) qv[i] = *reinterpret_cast<const ulonglong2*>(tb + DK + i * 32 + rg * 4);
        fetch(min(tq + j + 1, n - 1));
        float r0 = sum2(add2(a0, b0)), r1 = sum2(add2(a1, b1));
#pragma unroll
        for (int o = 1; o < 8; o <<= 1) {
          r0 += __shfl_xor_sync(0xffffffffu, r0, o);
          r1 += __shfl_xor_sync(0xffffffffu, r1, o);
        }
        const float u0 = beta * (v.x - r0), u1 = beta * (v.y - r1);
        const f32x2 uu0 = pack2(u0, u0), uu1 = pack2(u1, u1);
        a0 = a1 = b0 = b1 = 0;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          s0[i * 2] = fma2(kk[i * 2], uu0, s0[i * 2]);
          s1[i * 2] = fma2(kk[i * 2], uu1, s1[i * 2]);
          s0[i * 2 + 1] = fma2(kk[i * 2 + 1], uu0, s0[i * 2 + 1]);
          s1[i * 2 + 1] = fma2(kk[i * 2 + 1], uu1, s1[i * 2 + 1]);
          a0 = fma2(s0[i * 2], qv[i].x, a0);
          a1 = fma2(s1[i * 2], qv[i].x, a1);
          b0 = fma2(s0[i * 2 + 1], qv[i].y, b0);
          b1 = fma2(s1[i * 2 + 1], qv[i].y, b1);
        }
        part[2 * j] = sum2(add2(a0, b0));
        part[2 * j + 1] = sum2(add2(a1, b1));
      }
      // the eight lanes of a column pair add their parts: every exchange halves the values a lane keeps,
      // and lane rg ends with token tq + rg / 2, column rg % 2
#pragma unroll
      for (int o = 4, cnt = 4; o > 0; o >>= 1, cnt >>= 1) {
        const bool up = (rg & o) != 0;
#pragma unroll
        for (int i = 0; i < cnt; ++i) {
          const float keep = up ? part[i + cnt] : part[i], give = up ? part[i] : part[i + cnt];
          part[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
      }
      const int tk = tq + (rg >> 1);
      if (live && tk < n) op[static_cast<long long>(tk) * p.h * p.dv + (rg & 1)] = part[0];
    }
    __syncthreads();
  }
  if (slot >= 0 && live) {
#pragma unroll
    for (int i = 0; i < NR; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        float2 a, b;
        unpack2(s0[i * 2 + j], a.x, b.x);
        unpack2(s1[i * 2 + j], a.y, b.y);
        float* rp = sp + static_cast<long long>(i * 32 + rg * 4 + j * 2) * p.dv;
        *reinterpret_cast<float2*>(rp) = a;
        *reinterpret_cast<float2*>(rp + p.dv) = b;
      }
  }
}

// One warp per (token, head): out = o / rms(o) * w * sigmoid(gate)
template <typename T>
__global__ void __launch_bounds__(256) delta_gate_kernel(const DeltaParams p) {
  pdl_wait();
  pdl_trigger();
  const long long w = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= static_cast<long long>(p.tokens) * p.h) return;
  const int head = static_cast<int>(w % p.h);
  const long long t = w / p.h;
  const float* o = p.o + w * p.dv;
  float sq = 0.f;
  for (int e = lane * 4; e < p.dv; e += 128) {
    float v[4];
    ld4(o + e, v);
#pragma unroll
    for (int i = 0; i < 4; ++i) sq += v[i] * v[i];
  }
  const float inv = 1.f / sqrtf(warp_sum(sq) / p.dv_true + p.eps);
  const T* gr = static_cast<const T*>(p.z) + t * p.ldz + p.gate_off + head * p.dv;
  T* out = static_cast<T*>(p.out) + w * p.dv;
  for (int e = lane * 4; e < p.dv; e += 128) {
    float v[4], g[4], n[4];
    ld4(o + e, v);
    ld4(gr + e, g);
    ld4(p.norm_w + e, n);
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = v[i] * inv * n[i] * sigmoid_f32(g[i]);
    st4(out + e, v);
  }
}

// Decode. grid: (h, seqs); threads = (dv / 4) * ceil(dk / NRT): thread (cg, rg) owns four columns of
// NRT rows. Dynamic shared memory: (3 dk + (rgs + 1) dv + 32) floats.
constexpr int kStepThreads = 768;   // most threads of a decode block; larger heads are scanned

// kMax: most threads of this instance (two blocks of up to 512 share an SM, so that one loads while the
// other computes)
template <typename T, int NRT, int kMax>
__global__ void __launch_bounds__(kMax, kMax <= 512 ? 2 : 1) delta_step_kernel(const DeltaParams p) {
  extern __shared__ __align__(16) float sm[];
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int cgs = p.dv >> 2, cg = tid % cgs, rg = tid / cgs, rgs = blockDim.x / cgs;
  const bool worker = rg < rgs;
  const int slot = p.slots[seq];
  const bool carried = slot >= 0 && p.positions[seq] > 0;
  float4* sp = reinterpret_cast<float4*>(p.state + (static_cast<long long>(slot < 0 ? 0 : slot) * p.h + head) * p.dk * p.dv) + cg;
  // the state was last written by an earlier step, not by the kernel right before this one: its load
  // does not have to wait for that kernel
  float4 s[NRT];
#pragma unroll
  for (int i = 0; i < NRT; ++i) {
    const int r = rg * NRT + i;
    s[i] = carried && worker && r < p.dk ? sp[static_cast<long long>(r) * cgs] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  pdl_trigger();
  float *ks = sm, *qs = sm + p.dk, *gs = sm + 2 * p.dk, *us = sm + 3 * p.dk, *part = us + p.dv, *red = part + rgs * p.dv;
  const int kh = head / (p.h / p.hk);
  const long long kb = (static_cast<long long>(seq) * p.hk + kh) * p.dk, gb = (static_cast<long long>(seq) * p.h + head) * p.dk;
  for (int i = tid; i < p.dk; i += blockDim.x) {
    ks[i] = p.k[kb + i];
    qs[i] = p.q[kb + i];
    gs[i] = p.g[gb + i];
  }
  __syncthreads();
  if (worker) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NRT; ++i) {
      const int r = rg * NRT + i;
      if (r < p.dk) {
        const float g = gs[r], k = ks[r];
        s[i].x *= g; s[i].y *= g; s[i].z *= g; s[i].w *= g;
        a.x += s[i].x * k; a.y += s[i].y * k; a.z += s[i].z * k; a.w += s[i].w * k;
      }
    }
    reinterpret_cast<float4*>(part + rg * p.dv)[cg] = a;
  }
  __syncthreads();
  const long long ob = (static_cast<long long>(seq) * p.h + head) * p.dv;
  for (int c = tid; c < p.dv; c += blockDim.x) {
    float m = 0.f;
    for (int r = 0; r < rgs; ++r) m += part[r * p.dv + c];
    us[c] = p.beta[static_cast<long long>(seq) * p.h + head] * (p.v[ob + c] - m);
  }
  __syncthreads();
  if (worker) {
    const float4 u = reinterpret_cast<const float4*>(us)[cg];
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NRT; ++i) {
      const int r = rg * NRT + i;
      if (r < p.dk) {
        const float k = ks[r], q = qs[r];
        s[i].x += k * u.x; s[i].y += k * u.y; s[i].z += k * u.z; s[i].w += k * u.w;
        a.x += s[i].x * q; a.y += s[i].y * q; a.z += s[i].z * q; a.w += s[i].w * q;
        if (slot >= 0) sp[static_cast<long long>(r) * cgs] = s[i];
      }
    }
    reinterpret_cast<float4*>(part + rg * p.dv)[cg] = a;
  }
  __syncthreads();
  // blockDim >= dv: one thread per output value
  float o = 0.f;
  if (tid < p.dv)
    for (int r = 0; r < rgs; ++r) o += part[r * p.dv + tid];
  float sq = warp_sum(tid < p.dv ? o * o : 0.f);
  if ((tid & 31) == 0) red[tid >> 5] = sq;
  __syncthreads();
  if (tid < p.dv) {
    sq = 0.f;
    for (int i = 0; i * 32 < p.dv; ++i) sq += red[i];
    const float gate = ld1(static_cast<const T*>(p.z) + seq * p.ldz + p.gate_off + head * p.dv + tid);
    const float y = o / sqrtf(sq / p.dv_true + p.eps) * __bfloat162float(p.norm_w[tid]) * sigmoid_f32(gate);
    static_cast<T*>(p.out)[ob + tid] = static_cast<T>(y);
  }
}

template <int NR>
cudaError_t launch_scan(const DeltaParams& p, cudaStream_t stream) {
  const int smem = 2 * kScanTokens * (3 * NR * 32 + kScanCols + 4) * 4;
  static PerDeviceOnce once;
  if (once.first_time()) cudaFuncSetAttribute(delta_scan_kernel<NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  // an ordinary launch: blocks that were started while the last blocks of the kernel before still run would crowd the
  // processors that are free first, and there are few blocks
  delta_scan_kernel<NR><<<dim3((p.dv + kScanCols - 1) / kScanCols, p.h, p.seqs), 128, smem, stream>>>(p);
  return cudaGetLastError();
}

template <typename T, int NRT, int kMax>
cudaError_t launch_step_of(const DeltaParams& p, int threads, cudaStream_t stream) {
  const int rgs = threads / (p.dv / 4);
  const int smem = (3 * p.dk + (rgs + 1) * p.dv + 32) * 4;
  static PerDeviceOnce once;
  if (once.first_time()) cudaFuncSetAttribute(delta_step_kernel<T, NRT, kMax>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
  return launch_pdl(delta_step_kernel<T, NRT, kMax>, dim3(p.h, p.seqs), dim3(threads), smem, stream, p);
}

template <typename T, int NRT>
cudaError_t launch_step(const DeltaParams& p, int threads, cudaStream_t stream) {
  return threads <= 512 ? launch_step_of<T, NRT, 512>(p, threads, stream) : launch_step_of<T, NRT, kStepThreads>(p, threads, stream);
}

template <typename T>
int delta_impl(const DeltaParams& p, cudaStream_t stream) {
  const bool decode = p.cu_q == nullptr;
  cudaError_t e;
  if (p.taps == 4 && p.dk <= 128) {
    const int slices = 2 * p.hk + (p.h * p.dv + 127) / 128 + (p.h * p.dk + 127) / 128;
    const int run = decode || static_cast<long long>(p.tokens) * slices < 148 * 64 * 8 ? 1 : 8;
    e = launch_pdl(delta_prep4_kernel<T>, dim3((p.tokens + 8 * run - 1) / (8 * run), slices), dim3(256), 0, stream, p, run);
  } else {
    e = launch_pdl(delta_prep_kernel<T>, dim3((p.tokens + 7) / 8, 2 * p.hk + 2 * p.h), dim3(256), 0, stream, p);
  }
  if (e != cudaSuccess) return -static_cast<int>(e) - 300;
  if (decode) {
    const int cgs = p.dv / 4;
    int nrt = 8;
    int threads = cgs * ((p.dk + nrt - 1) / nrt);
    while (nrt > 2 && threads < 128) { nrt /= 2; threads = cgs * ((p.dk + nrt - 1) / nrt); }
    if (threads < p.dv) threads = p.dv;
    threads = (threads + 31) / 32 * 32;
    if (threads <= kStepThreads) {
      switch (nrt) {
        case 8: e = launch_step<T, 8>(p, threads, stream); break;
        case 4: e = launch_step<T, 4>(p, threads, stream); break;
        default: e = launch_step<T, 2>(p, threads, stream); break;
      }
      return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
    }
  } else {
    if (p.taps > 1) {
      const int channels = 2 * p.hk * p.dk + p.h * p.dv;
      e = launch_pdl(delta_tail_kernel<T>, dim3((channels + 255) / 256, p.seqs), dim3(256), 0, stream, p);
      if (e != cudaSuccess) return -static_cast<int>(e) - 300;
    }
  }
  switch (p.dk / 32) {
    case 1: e = launch_scan<1>(p, stream); break;
    case 2: e = launch_scan<2>(p, stream); break;
    case 3: e = launch_scan<3>(p, stream); break;
    case 4: e = launch_scan<4>(p, stream); break;
    case 5: e = launch_scan<5>(p, stream); break;
    case 6: e = launch_scan<6>(p, stream); break;
    case 7: e = launch_scan<7>(p, stream); break;
    default: e = launch_scan<8>(p, stream); break;
  }
  if (e != cudaSuccess) return -static_cast<int>(e) - 300;
  const long long warps = static_cast<long long>(p.tokens) * p.h;
  e = launch_pdl(delta_gate_kernel<T>, dim3(static_cast<unsigned>((warps + 7) / 8)), dim3(256), 0, stream, p);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

}  // namespace b200

using namespace b200;

// fp32 scratch of one call, in bytes (q, k, v, g, beta, o)
B200_API long long b200_delta_workspace_bytes(int tokens, int h, int hk, int dk, int dv) {
  const long long per = 2ll * hk * dk + 2ll * h * dv + static_cast<long long>(h) * dk + (h + 3) / 4 * 4;
  return per * tokens * 4;
}

// Number of kernels one call launches (for the launch count)
B200_API int b200_delta_launches(int decode, int taps, int dk, int dv) {
  if (decode) return (dv / 4) * ((dk + 7) / 8) <= kStepThreads && dv <= kStepThreads ? 2 : 3;
  return taps > 1 ? 4 : 3;
}

// See the header comment and DeltaParams. dk (<= 256) a multiple of 32, dv a multiple of 8; dk_true /
// dv_true are the sizes before padding (the q scale and the output norm use them; padded channels
// carry zeros). cu_q null: one token per sequence (decode).
B200_API int b200_delta(const void* proj, const void* z, const float* conv_w, const float* a, const float* dt_bias,
                        void* conv_state, void* state, const void* norm_w, const int* positions, const int* cu_q,
                        const int* slots, void* workspace, void* out, int tokens, int seqs, int h, int hk, int dk, int dv,
                        int dk_true, int dv_true, int taps, long long ldp, int b_off, long long ldz, int gate_off, float eps,
                        int f32, cudaStream_t stream) {
  if (tokens <= 0 || seqs <= 0) return 0;
  if (dk % 32 || dk < 32 || dk > kDeltaMaxDk || dv % 8 || dv < 8 || dv > 1024 || hk < 1 || h % hk || taps < 1) return -2;
  if (ldp % 8 || ldz % 8 || gate_off % 8 || seqs > 65535 || h > 65535) return -2;
  if (!cu_q && tokens != seqs) return -2;
  DeltaParams p{};
  p.proj = proj; p.z = z; p.conv_w = conv_w; p.a = a; p.dt_bias = dt_bias;
  p.conv_state = conv_state; p.state = static_cast<float*>(state); p.norm_w = static_cast<const __nv_bfloat16*>(norm_w);
  p.positions = positions; p.cu_q = cu_q; p.slots = slots;
  p.out = out; p.ldp = ldp; p.ldz = ldz;
  p.tokens = tokens; p.seqs = seqs; p.h = h; p.hk = hk; p.dk = dk; p.dv = dv; p.taps = taps; p.b_off = b_off;
  p.gate_off = gate_off; p.dv_true = dv_true; p.eps = eps;
  p.q_scale = 1.f / sqrtf(static_cast<float>(dk_true));
  float* ws = static_cast<float*>(workspace);
  const long long t = tokens;
  p.q = ws; ws += t * hk * dk;
  p.k = ws; ws += t * hk * dk;
  p.v = ws; ws += t * h * dv;
  p.g = ws; ws += t * h * dk;
  p.o = ws; ws += t * h * dv;
  p.beta = ws;
  return f32 ? delta_impl<float>(p, stream) : delta_impl<__nv_bfloat16>(p, stream);
}
