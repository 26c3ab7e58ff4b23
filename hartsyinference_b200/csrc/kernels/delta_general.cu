// Delta-rule mixer whose removal has a rate of its own per key channel.
//
// Per head and sequence a matrix S [dk][dv] in fp32, updated by every token t from the state before it:
//   S_t = Diag(e_t) S - (a_t u_t) (u_t^T S) + k_t v_t^T;   o_t = S_t^T r_t
//   y_t = sigmoid(gate_t) w o_t / rms(o_t)
// u is k as a unit vector, e = exp(-exp(-1/2) sigmoid(z + decay_bias)), a = sigmoid(logit + rate_bias). Both products
// with the state read the old one:
//   p = S^T u,  s = S^T (e r);   S_t = e S - (a u) p^T + u (|k| v)^T;   o = s - p ((a u) r) + |k| v (u r)
// so a token costs one pass of reductions over the rows instead of two that wait for each other.
//
//  * general_prep   one warp per (token, head): unit key, decay, removal and read vectors and both dot products as one
//                   fp32 record.
//  * general_scan   portions of prompts: the columns of S are independent, a block takes 32 of them (a thread keeps four
//                   columns of an eighth of the rows in registers) and walks over the tokens, whose records are staged
//                   through shared memory. The operations do not depend on where a prompt is cut.
//  * general_gate   the output norm and gate of a scanned portion, one warp per (token, head).
//  * general_step   decode: one block per (sequence, head) forms its own record, reads the state once, applies the
//                   update, writes it back and emits the normed, gated output: one launch.
//
// State lives in slots, [slots][heads][dk][dv] fp32; a sequence whose portion starts at position 0 starts from zeros
// whatever its slot held before, a negative slot is computed from zeros and stored nowhere.
#include "mixer_common.cuh"

namespace b200 {

struct GeneralDeltaParams {
  const void* proj;          // [T][ldp]: r | k | removal logits (h * dk each) | v | gate logits (h * dv each)
  const void* z;             // [T][ldz]: decay logits (h * dk)
  const float *decay_bias, *rate_bias;   // [h * dk]
  const __nv_bfloat16* norm_w;           // [h * dv]
  float* state;              // [slots][h][dk][dv]
  const int* positions;      // [T]
  const int* cu_q;           // [seqs + 1]; null: one token per sequence
  const int* slots;          // [seqs]
  float *rec, *o;            // scratch: [T][h][4 + 4 dk + dv], [T][h][dv]
  void* out;                 // [T][ldo]
  long long ldp, ldz, ldo;
  int tokens, seqs, h, dk, dv, d_true;
  int longest;               // tokens of the longest portion (0: not known)
  float eps;
};

constexpr int kGenMaxD = 256;
constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ float general_decay(float z) { return decay_of(0.60653065971263342f * sigmoid_f32(z)); }   // exp(-1/2)

// Record of one token and head: {(a u) r, u r, 0, 0} | u | e | a u | e r | |k| v
__host__ __device__ inline int record_floats(int dk, int dv) { return 4 + 4 * dk + dv; }

template <typename T>
__global__ void __launch_bounds__(256) general_prep_kernel(const GeneralDeltaParams p) {
  pdl_wait();
  pdl_trigger();
  const long long w = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= static_cast<long long>(p.tokens) * p.h) return;
  const int head = static_cast<int>(w % p.h), n = p.h * p.dk;
  const long long t = w / p.h;
  const T* row = static_cast<const T*>(p.proj) + t * p.ldp + head * p.dk;
  const T* zr = static_cast<const T*>(p.z) + t * p.ldz + head * p.dk;
  float* rec = p.rec + w * record_floats(p.dk, p.dv);
  constexpr int kIt = kGenMaxD / 128;
  float k[kIt][4], sq = 0.f;
#pragma unroll
  for (int i = 0; i < kIt; ++i) {
    const int e = lane * 4 + i * 128;
#pragma unroll
    for (int j = 0; j < 4; ++j) k[i][j] = 0.f;
    if (e < p.dk) ld4(row + n + e, k[i]);
#pragma unroll
    for (int j = 0; j < 4; ++j) sq = fmaf(k[i][j], k[i][j], sq);
  }
  const float len = sqrtf(warp_sum(sq) + kUnitEps), inv = 1.f / len;
  float c1 = 0.f, c2 = 0.f;
#pragma unroll
  for (int i = 0; i < kIt; ++i) {
    const int e = lane * 4 + i * 128;
    if (e >= p.dk) continue;
    float r[4], a[4], z[4], ab[4], zb[4], u[4], er[4];
    ld4(row + e, r);
    ld4(row + 2 * n + e, a);
    ld4(zr + e, z);
    ld4(p.rate_bias + head * p.dk + e, ab);
    ld4(p.decay_bias + head * p.dk + e, zb);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      u[j] = k[i][j] * inv;
      z[j] = general_decay(z[j] + zb[j]);
      a[j] = sigmoid_f32(a[j] + ab[j]) * u[j];
      er[j] = z[j] * r[j];
      c1 = fmaf(a[j], r[j], c1);
      c2 = fmaf(u[j], r[j], c2);
    }
    st4(rec + 4 + e, u);
    st4(rec + 4 + p.dk + e, z);
    st4(rec + 4 + 2 * p.dk + e, a);
    st4(rec + 4 + 3 * p.dk + e, er);
  }
  c1 = warp_sum(c1);
  c2 = warp_sum(c2);
  if (lane == 0) {
    const float c[4] = {c1, c2, 0.f, 0.f};
    st4(rec, c);
  }
  const T* vr = static_cast<const T*>(p.proj) + t * p.ldp + 3 * n + head * p.dv;
  for (int e = lane * 4; e < p.dv; e += 128) {
    float v[4];
    ld4(vr + e, v);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] *= len;
    st4(rec + 4 + 4 * p.dk + e, v);
  }
}

constexpr int kGenTokens = 8;      // tokens per staging buffer
constexpr int kGenCols = 32;       // columns of S per block
constexpr int kGenFew = 1200;      // fewer blocks than this: more lanes per column

// grid: (ceil(dv / 32), h, seqs), 8 RL threads. dk = 4 RL NV. A column's rows are dealt over RL lanes (8, or 16 for more
// warps when there are few columns). Lane: rows 4 (i RL + lane % RL) + 0..3 of columns 4 (lane / RL) + 0..3 of the warp's:
// four columns share what a lane reads from shared memory.
template <int NV, int RL>
__global__ void __launch_bounds__(8 * RL) general_scan_kernel(const GeneralDeltaParams p) {
  constexpr int DK = NV * RL * 4, NR = NV, kStep = 4 * RL, kThreads = 8 * RL;
  constexpr int kTok = 4 + 4 * DK + kGenCols;       // floats per staged token
  extern __shared__ __align__(16) float sm[];
  const int head = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int rg = tid % RL;
  const int col0 = blockIdx.x * kGenCols, lc = tid / RL * 4, col = col0 + lc;
  const int first = p.cu_q ? p.cu_q[seq] : seq;
  const int len = p.cu_q ? p.cu_q[seq + 1] - first : 1;
  if (len <= 0) return;
  const int slot = p.slots[seq];
  const bool carried = slot >= 0 && p.positions[first] > 0;
  const bool live = col < p.dv;
  float* sp = p.state + (static_cast<long long>(slot < 0 ? 0 : slot) * p.h + head) * DK * p.dv + col;
  const int rec = record_floats(DK, p.dv);

  f32x2 s[4][NR * 2];                 // four columns, row pairs
#pragma unroll
  for (int i = 0; i < NR; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
      if (carried && live) {
        const float* rp = sp + static_cast<long long>(i * kStep + rg * 4 + j * 2) * p.dv;
        ld4(rp, a);
        ld4(rp + p.dv, b);
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) s[c][i * 2 + j] = pack2(a[c], b[c]);
    }

  auto stage = [&](int t0, int buf) {
    float* base = sm + buf * kGenTokens * kTok;
    const int n = min(kGenTokens, len - t0);
    constexpr int kVec = kTok / 4;
    for (int i = tid; i < n * kVec; i += kThreads) {
      const int tk = i / kVec, c = (i - tk * kVec) * 4;
      const float* src = p.rec + (static_cast<long long>(first + t0 + tk) * p.h + head) * rec;
      const bool value = c >= 4 + 4 * DK;
      const bool ok = !value || col0 + c - (4 + 4 * DK) < p.dv;
      copy_async_16(smem_u32(base + tk * kTok + c), ok ? src + c + (value ? col0 : 0) : p.rec, ok);
    }
  };
  auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };

  stage(0, 0);
  commit();
  int buf = 0;
  for (int t0 = 0; t0 < len; t0 += kGenTokens, buf ^= 1) {
    if (t0 + kGenTokens < len) stage(t0 + kGenTokens, buf ^ 1);
    commit();
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const int n = min(kGenTokens, len - t0);
    const float* base = sm + buf * kGenTokens * kTok;
    float* op = p.o + (static_cast<long long>(first + t0) * p.h + head) * p.dv + col;
    ulonglong2 nu[NR], ner[NR];            // the next token's u and e r, read while the current one is computed
    auto fetch = [&](int tk) {
      const float* rows = base + tk * kTok + 4 + rg * 4;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        nu[i] = *reinterpret_cast<const ulonglong2*>(rows + i * kStep);
        ner[i] = *reinterpret_cast<const ulonglong2*>(rows + 3 * DK + i * kStep);
      }
    };
    fetch(0);
    for (int tq = 0; tq < n; tq += 4) {
      float part[16];                      // outputs of four tokens x four columns, this lane's rows
#pragma unroll
      for (int j = 0; j < 4; ++j) {
#pragma unroll
        for (int c = 0; c < 4; ++c) part[4 * j + c] = 0.f;
        if (tq + j >= n) continue;
        const float* tb = base + (tq + j) * kTok;
        const float* rows = tb + 4 + rg * 4;
        ulonglong2 uu[NR];
        f32x2 a[4], b[4], x[4], y[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) a[c] = b[c] = x[c] = y[c] = 0;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          uu[i] = nu[i];
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            a[c] = fma2(s[c][i * 2], uu[i].x, a[c]);
            b[c] = fma2(s[c][i * 2 + 1], uu[i].y, b[c]);
          }
        }
        float r[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) r[c] = sum2(add2(a[c], b[c]));
#pragma unroll
        for (int o = 1; o < RL; o <<= 1)
#pragma unroll
          for (int c = 0; c < 4; ++c) r[c] += __shfl_xor_sync(0xffffffffu, r[c], o);
#pragma unroll
        for (int i = 0; i < NR; ++i)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            x[c] = fma2(s[c][i * 2], ner[i].x, x[c]);
            y[c] = fma2(s[c][i * 2 + 1], ner[i].y, y[c]);
          }
        fetch(min(tq + j + 1, n - 1));
        const float2 k = *reinterpret_cast<const float2*>(tb);
        float v[4];
        ld4(tb + 4 + 4 * DK + lc, v);
#pragma unroll
        for (int i = 0; i < NR; ++i) {     // what does not need the reads: decay and the new value
          const ulonglong2 e = *reinterpret_cast<const ulonglong2*>(rows + DK + i * kStep);
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const f32x2 vc = pack2(v[c], v[c]);
            s[c][i * 2] = fma2(uu[i].x, vc, mul2(e.x, s[c][i * 2]));
            s[c][i * 2 + 1] = fma2(uu[i].y, vc, mul2(e.y, s[c][i * 2 + 1]));
          }
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          part[4 * j + c] = sum2(add2(x[c], y[c]));
          if (rg == 0) part[4 * j + c] += v[c] * k.y - r[c] * k.x;     // what the token itself adds, once per column
          r[c] = -r[c];
        }
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          const ulonglong2 au = *reinterpret_cast<const ulonglong2*>(rows + 2 * DK + i * kStep);
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const f32x2 rc = pack2(r[c], r[c]);
            s[c][i * 2] = fma2(au.x, rc, s[c][i * 2]);
            s[c][i * 2 + 1] = fma2(au.y, rc, s[c][i * 2 + 1]);
          }
        }
      }
      // the lanes of four columns add their parts: every exchange halves the values a lane keeps, and lane rg ends with
      // one of the sixteen, or two neighbours
#pragma unroll
      for (int o = RL / 2, cnt = 8; o > 0; o >>= 1, cnt >>= 1) {
        const bool up = (rg & o) != 0;
#pragma unroll
        for (int i = 0; i < cnt; ++i) {
          const float keep = up ? part[i + cnt] : part[i], give = up ? part[i] : part[i + cnt];
          part[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
      }
      const int at = rg * (16 / RL), tk = tq + (at >> 2);
      if (live && tk < n) {
        float* dst = op + static_cast<long long>(tk) * p.h * p.dv + (at & 3);
        if (RL == 8) *reinterpret_cast<float2*>(dst) = make_float2(part[0], part[1]);
        else *dst = part[0];
      }
    }
    __syncthreads();
  }
  if (slot >= 0 && live) {
#pragma unroll
    for (int i = 0; i < NR; ++i)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        float a[4], b[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) unpack2(s[c][i * 2 + j], a[c], b[c]);
        float* rp = sp + static_cast<long long>(i * kStep + rg * 4 + j * 2) * p.dv;
        st4(rp, a);
        st4(rp + p.dv, b);
      }
  }
}

// One warp per (token, head): out = o / rms(o) * w * sigmoid(gate)
template <typename T>
__global__ void __launch_bounds__(256) general_gate_kernel(const GeneralDeltaParams p) {
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
  const float inv = 1.f / sqrtf(warp_sum(sq) / p.d_true + p.eps);
  const T* gr = static_cast<const T*>(p.proj) + t * p.ldp + 3 * p.h * p.dk + p.h * p.dv + head * p.dv;
  T* out = static_cast<T*>(p.out) + t * p.ldo + head * p.dv;
  for (int e = lane * 4; e < p.dv; e += 128) {
    float v[4], g[4], n[4];
    ld4(o + e, v);
    ld4(gr + e, g);
    ld4(p.norm_w + head * p.dv + e, n);
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = v[i] * inv * n[i] * sigmoid_f32(g[i]);
    st4(out + e, v);
  }
}

// Decode. grid: (h, seqs); threads = (dv / 4) * ceil(dk / NRT), at least dk and dv: thread (cg, rg) owns four columns of
// NRT rows. Dynamic shared memory: (4 dk + dv + 2 rgs dv + 96) floats.
constexpr int kGenStepThreads = 768;   // most threads of a decode block; larger heads are scanned

template <typename T, int NRT, int kMax>
__global__ void __launch_bounds__(kMax, kMax <= 512 ? 2 : 1) general_step_kernel(const GeneralDeltaParams p) {
  extern __shared__ __align__(16) float sm[];
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, dk = p.dk, dv = p.dv;
  const int cgs = dv >> 2, cg = tid % cgs, rg = tid / cgs, rgs = blockDim.x / cgs;
  const bool worker = rg < rgs;
  const int slot = p.slots[seq];
  const bool carried = slot >= 0 && p.positions[seq] > 0;
  float4* sp = reinterpret_cast<float4*>(p.state + (static_cast<long long>(slot < 0 ? 0 : slot) * p.h + head) * dk * dv) + cg;
  // the state was last written by an earlier step, not by the kernel right before this one: its load does not have to
  // wait for that kernel
  float4 s[NRT];
#pragma unroll
  for (int i = 0; i < NRT; ++i) {
    const int r = rg * NRT + i;
    s[i] = carried && worker && r < dk ? sp[static_cast<long long>(r) * cgs] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float zb = 0.f, ab = 0.f;
  if (tid < dk) {
    zb = p.decay_bias[head * dk + tid];
    ab = p.rate_bias[head * dk + tid];
  }
  pdl_wait();
  pdl_trigger();
  float *us = sm, *es = sm + dk, *as = sm + 2 * dk, *ers = sm + 3 * dk, *vs = sm + 4 * dk;
  float *pp = vs + dv, *ps = pp + rgs * dv, *red = ps + rgs * dv;      // red: three rows of one value per warp
  const int n = p.h * dk, warp = tid >> 5, warps = (blockDim.x + 31) >> 5;
  const T* row = static_cast<const T*>(p.proj) + static_cast<long long>(seq) * p.ldp;
  float k = 0.f, r = 0.f, e = 0.f, a = 0.f, v = 0.f;
  if (tid < dk) {
    k = ld1(row + n + head * dk + tid);
    r = ld1(row + head * dk + tid);
    a = sigmoid_f32(ld1(row + 2 * n + head * dk + tid) + ab);
    e = general_decay(ld1(static_cast<const T*>(p.z) + seq * p.ldz + head * dk + tid) + zb);
  }
  if (tid < dv) v = ld1(row + 3 * n + head * dv + tid);
  float q = warp_sum(k * k), c1 = warp_sum(a * k * r), c2 = warp_sum(k * r);
  if ((tid & 31) == 0) {
    red[warp] = q;
    red[32 + warp] = c1;
    red[64 + warp] = c2;
  }
  __syncthreads();
  q = c1 = c2 = 0.f;
  for (int i = 0; i < warps; ++i) {
    q += red[i];
    c1 += red[32 + i];
    c2 += red[64 + i];
  }
  const float len = sqrtf(q + kUnitEps), inv = 1.f / len;
  c1 *= inv;
  c2 *= inv;
  if (tid < dk) {
    us[tid] = k * inv;
    es[tid] = e;
    as[tid] = a * k * inv;
    ers[tid] = e * r;
  }
  if (tid < dv) vs[tid] = v * len;
  __syncthreads();
  if (worker) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
#pragma unroll
    for (int i = 0; i < NRT; ++i) {
      const int at = rg * NRT + i;
      if (at < dk) {
        const float u = us[at], er = ers[at];
        x.x += s[i].x * u; x.y += s[i].y * u; x.z += s[i].z * u; x.w += s[i].w * u;
        y.x += s[i].x * er; y.y += s[i].y * er; y.z += s[i].z * er; y.w += s[i].w * er;
      }
    }
    reinterpret_cast<float4*>(pp + rg * dv)[cg] = x;
    reinterpret_cast<float4*>(ps + rg * dv)[cg] = y;
  }
  __syncthreads();
  float o = 0.f, read = 0.f;
  if (tid < dv) {
    for (int i = 0; i < rgs; ++i) {
      read += pp[i * dv + tid];
      o += ps[i * dv + tid];
    }
    o += vs[tid] * c2 - read * c1;
  }
  const float sq = warp_sum(o * o);
  __syncthreads();                     // the sums of pp are read, the totals in red too
  if (tid < dv) pp[tid] = read;
  if ((tid & 31) == 0) red[warp] = sq;
  __syncthreads();
  if (worker && slot >= 0) {
    const float4 x = reinterpret_cast<const float4*>(pp)[cg], w = reinterpret_cast<const float4*>(vs)[cg];
#pragma unroll
    for (int i = 0; i < NRT; ++i) {
      const int at = rg * NRT + i;
      if (at < dk) {
        const float u = us[at], d = es[at], m = -as[at];
        sp[static_cast<long long>(at) * cgs] =
            make_float4(fmaf(m, x.x, fmaf(u, w.x, d * s[i].x)), fmaf(m, x.y, fmaf(u, w.y, d * s[i].y)),
                        fmaf(m, x.z, fmaf(u, w.z, d * s[i].z)), fmaf(m, x.w, fmaf(u, w.w, d * s[i].w)));
      }
    }
  }
  if (tid < dv) {
    float total = 0.f;
    for (int i = 0; i < warps; ++i) total += red[i];
    const float gate = ld1(row + 3 * n + p.h * dv + head * dv + tid);
    const float y = o / sqrtf(total / p.d_true + p.eps) * __bfloat162float(p.norm_w[head * dv + tid]) * sigmoid_f32(gate);
    static_cast<T*>(p.out)[seq * p.ldo + head * dv + tid] = static_cast<T>(y);
  }
}

// An ordinary launch: blocks that were started while the last blocks of the kernel before still run would crowd the
// processors that are free first, and there are few blocks.
template <int NV, int RL>
cudaError_t launch_general_scan(const GeneralDeltaParams& p, cudaStream_t stream) {
  const int smem = 2 * kGenTokens * (4 + 16 * NV * RL + kGenCols) * 4;
  static PerDeviceOnce once;
  if (once.first_time()) cudaFuncSetAttribute(general_scan_kernel<NV, RL>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  general_scan_kernel<NV, RL><<<dim3((p.dv + kGenCols - 1) / kGenCols, p.h, p.seqs), 8 * RL, smem, stream>>>(p);
  return cudaGetLastError();
}

template <typename T, int NRT, int kMax>
cudaError_t launch_general_step_of(const GeneralDeltaParams& p, int threads, cudaStream_t stream) {
  const int rgs = threads / (p.dv / 4);
  const int smem = (4 * p.dk + p.dv + 2 * rgs * p.dv + 96) * 4;
  static PerDeviceOnce once;
  if (once.first_time()) cudaFuncSetAttribute(general_step_kernel<T, NRT, kMax>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
  return launch_pdl(general_step_kernel<T, NRT, kMax>, dim3(p.h, p.seqs), dim3(threads), smem, stream, p);
}

template <typename T, int NRT>
cudaError_t launch_general_step(const GeneralDeltaParams& p, int threads, cudaStream_t stream) {
  return threads <= 512 ? launch_general_step_of<T, NRT, 512>(p, threads, stream)
                        : launch_general_step_of<T, NRT, kGenStepThreads>(p, threads, stream);
}

// Threads of a decode block with nrt rows each
inline int general_step_threads(int dk, int dv, int nrt) {
  int threads = (dv / 4) * ((dk + nrt - 1) / nrt);
  threads = threads < dv ? dv : threads;
  threads = threads < dk ? dk : threads;
  return (threads + 31) / 32 * 32;
}

template <typename T>
int general_delta_impl(const GeneralDeltaParams& p, cudaStream_t stream) {
  cudaError_t e;
  if (p.cu_q == nullptr && general_step_threads(p.dk, p.dv, 8) <= kGenStepThreads) {
    int nrt = 8;
    while (nrt > 2 && (p.dv / 4) * ((p.dk + nrt - 1) / nrt) < 128) nrt /= 2;
    const int threads = general_step_threads(p.dk, p.dv, nrt);
    e = nrt == 8 ? launch_general_step<T, 8>(p, threads, stream)
                 : nrt == 4 ? launch_general_step<T, 4>(p, threads, stream) : launch_general_step<T, 2>(p, threads, stream);
    return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
  }
  const dim3 warps(static_cast<unsigned>((static_cast<long long>(p.tokens) * p.h + 7) / 8));
  e = launch_pdl(general_prep_kernel<T>, warps, dim3(256), 0, stream, p);
  if (e != cudaSuccess) return -static_cast<int>(e) - 300;
  // single tokens beside long portions are done soon: count the portions as if all were as long as the longest
  const int portions = p.longest > 0 ? (p.tokens + p.longest - 1) / p.longest : p.seqs;
  const bool few = static_cast<long long>((p.dv + kGenCols - 1) / kGenCols) * p.h * portions < kGenFew;
  switch (p.dk / 32) {
    case 1: e = launch_general_scan<1, 8>(p, stream); break;
    case 2: e = few ? launch_general_scan<1, 16>(p, stream) : launch_general_scan<2, 8>(p, stream); break;
    case 3: e = launch_general_scan<3, 8>(p, stream); break;
    case 4: e = few ? launch_general_scan<2, 16>(p, stream) : launch_general_scan<4, 8>(p, stream); break;
    case 5: e = launch_general_scan<5, 8>(p, stream); break;
    case 6: e = few ? launch_general_scan<3, 16>(p, stream) : launch_general_scan<6, 8>(p, stream); break;
    case 7: e = launch_general_scan<7, 8>(p, stream); break;
    default: e = launch_general_scan<4, 16>(p, stream); break;
  }
  if (e != cudaSuccess) return -static_cast<int>(e) - 300;
  e = launch_pdl(general_gate_kernel<T>, warps, dim3(256), 0, stream, p);
  return e == cudaSuccess ? 0 : -static_cast<int>(e) - 300;
}

}  // namespace b200

using namespace b200;

// fp32 scratch of one call, in bytes (records, outputs before the norm)
B200_API long long b200_general_delta_workspace_bytes(int tokens, int h, int dk, int dv) {
  return static_cast<long long>(tokens) * h * (record_floats(dk, dv) + dv) * 4;
}

// Number of kernels one call launches (for the launch count)
B200_API int b200_general_delta_launches(int decode, int dk, int dv) {
  return decode && general_step_threads(dk, dv, 8) <= kGenStepThreads ? 1 : 3;
}

// See the header comment and GeneralDeltaParams. dk (<= 256) a multiple of 32, dv (<= 256) a multiple of 8; d_true is the
// head size before padding (the output norm uses it; padded channels carry zeros). cu_q null: one token per sequence.
// longest: tokens of the longest portion, 0 when not known.
B200_API int b200_general_delta(const void* proj, const void* z, const float* decay_bias, const float* rate_bias, const void* norm_w,
                                void* state, const int* positions, const int* cu_q, const int* slots, void* workspace, void* out,
                                int tokens, int seqs, int h, int dk, int dv, int d_true, long long ldp, long long ldz, long long ldo,
                                float eps, int longest, int f32, cudaStream_t stream) {
  if (tokens <= 0 || seqs <= 0) return 0;
  if (dk % 32 || dk < 32 || dk > kGenMaxD || dv % 8 || dv < 8 || dv > kGenMaxD || h < 1 || h > 65535 || seqs > 65535) return -2;
  if (ldp % 8 || ldz % 8 || ldo % 8 || ldp < 3ll * h * dk + 2ll * h * dv || (!cu_q && tokens != seqs)) return -2;
  GeneralDeltaParams p{};
  p.proj = proj; p.z = z; p.decay_bias = decay_bias; p.rate_bias = rate_bias;
  p.norm_w = static_cast<const __nv_bfloat16*>(norm_w);
  p.state = static_cast<float*>(state);
  p.positions = positions; p.cu_q = cu_q; p.slots = slots;
  p.rec = static_cast<float*>(workspace);
  p.o = p.rec + static_cast<long long>(tokens) * h * record_floats(dk, dv);
  p.out = out; p.ldp = ldp; p.ldz = ldz; p.ldo = ldo;
  p.tokens = tokens; p.seqs = seqs; p.h = h; p.dk = dk; p.dv = dv; p.d_true = d_true; p.eps = eps;
  p.longest = longest;
  return f32 ? general_delta_impl<float>(p, stream) : general_delta_impl<__nv_bfloat16>(p, stream);
}
