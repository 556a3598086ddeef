// Linear recurrences with a matrix state per head (sm_100a): gated delta rule with one decay per
// key channel, and the matrix memory with exponential gates (mLSTM).
//
//   delta_inputs    short causal convolution + SiLU of q, k, v, unit vectors, decays, step sizes
//   memory_inputs   q (scaled), k, v in fp32, log gates of the matrix memory
//   recurrent_scan  the recurrence itself, for every request of a step: portions of prompts and
//                   single tokens alike
//   head_norm_gate  o / rms(o) per head, times the norm weight, a sigmoid gate and a factor
//
// State of a request, addressed by its state slot, fp32 throughout:
//   matrix  [slot, head, vdim, DP]      S transposed: a value column's key entries are contiguous
//   vector  [slot, head, DP], scalar [slot, head]      (matrix memory: normaliser n, maximum m)
//   taps    [slot, taps, channels] in the model's type: row p % taps holds the convolution input
//           of position p.  A step reads the rows of positions in front of its portion before
//           the scan overwrites them.
// A portion that starts at position 0 starts from zeros whatever the slot holds, so slots need no
// clearing.  DP is the head dimension rounded up to 8 * RPL; the padding stays zero.
//
// The scan splits a head's value columns over threads: they are independent of each other.  Eight
// lanes share a column (RPL key rows each, in registers), CPT columns per lane group; a CTA holds a
// block of columns of one head of one request and walks its tokens in order, inputs staged through
// shared memory by cp.async one chunk ahead.  The result of a token does not depend on where the
// prompt was cut.
#include "common.cuh"

namespace b200 {
namespace recurrent {

constexpr unsigned int kKernelId = 80;
constexpr int kDelta = 0, kMemory = 1;

// fp32 pairs: two multiply-adds per instruction
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t both(float x) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %1};" : "=l"(d) : "f"(x));
  return d;
}
__device__ __forceinline__ float halves_sum(uint64_t x) {
  float lo, hi;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(x));
  return lo + hi;
}

__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) {
  return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)));
}

__device__ __forceinline__ void copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src)
               : "memory");
}
__device__ __forceinline__ void copy4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src)
               : "memory");
}
__device__ __forceinline__ void copy_commit() {
  asm volatile("cp.async.commit_group;" ::: "memory");
}
template <int N>
__device__ __forceinline__ void copy_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// Which tokens of the step belong to request r: [first, first + count).
struct Portion {
  int first, count;
};
__device__ __forceinline__ Portion portion_of(int r, int nd, const int* cu_q) {
  if (r < nd) return {r, 1};
  return {nd + cu_q[r - nd], cu_q[r - nd + 1] - cu_q[r - nd]};
}

// ---------------------------------------------------------------------------
struct DeltaIn {
  const void* x[3];          // q, k, v projections [T, channels] (views), row pitch ld
  const float* taps_w[3];    // [channels, taps] convolution weights, last column: current token
  const void* taps;          // state: [slots, taps, C] with C = all channels, q | k | v
  const float* z;            // [T, N * D] decay projection
  const float* bz;           // [T, N] step size projection
  const float* dt_bias;      // [N * D]
  const float* a_log;        // [N]
  float *q, *k;              // out: [T, G, DP]
  float *g;                  // out: [T, N, DP]
  float *v;                  // out: [T, N, VP]
  float *beta;               // out: [T, N]
  const long long* positions;
  const int* slots;          // [requests] state slots
  const int* cu_q;
  long long ld, ldz, ldb;
  int T, G, N, D, V, DP, VP, ntaps, num_slots, nd, np;
};

// Rows of the convolution window of one token: [o] = input of `o` tokens ago, null for none.
constexpr int kMaxTaps = 8;
template <typename T>
struct Window {
  const T* row[kMaxTaps];
};

template <typename T>
__device__ __forceinline__ float conv_silu(const Window<T>& w, const float* taps, int ntaps, int c) {
  float s = 0.0f;
#pragma unroll
  for (int o = kMaxTaps - 1; o >= 0; --o) {
    if (o >= ntaps || w.row[o] == nullptr) continue;
    s += taps[c * ntaps + (ntaps - 1 - o)] * to_f32<T>(w.row[o][c]);
  }
  return s / (1.0f + expf(-s));
}

template <typename T>
__global__ void __launch_bounds__(256) delta_inputs_kernel(const DeltaIn a) {
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int item = blockIdx.y * 8 + warp;          // [0, G): q and k heads; [G, G + N): v heads
  if (item >= a.G + a.N) return;
  const TokenPlace pl = token_place(t, a.nd, a.np, a.cu_q);
  if (pl.req < 0) return;
  const Portion po = portion_of(pl.req, a.nd, a.cu_q);
  const long long pos = a.positions[t];
  const int slot = a.slots[pl.req];
  const int C = 2 * a.G * a.D + a.N * a.V;
  auto window = [&](int which) {
    Window<T> w;
    const T* x = static_cast<const T*>(a.x[which]);
    const int off = which == 0 ? 0 : which == 1 ? a.G * a.D : 2 * a.G * a.D;
#pragma unroll
    for (int o = 0; o < kMaxTaps; ++o) {
      w.row[o] = nullptr;
      if (o >= a.ntaps || pos - o < 0) continue;
      if (t - o >= po.first) {
        w.row[o] = x + static_cast<long long>(t - o) * a.ld;
      } else if (slot >= 0 && slot < a.num_slots) {
        w.row[o] = static_cast<const T*>(a.taps) +
                   (static_cast<long long>(slot) * a.ntaps + (pos - o) % a.ntaps) * C + off;
      }
    }
    return w;
  };
  if (item < a.G) {
    constexpr int kMax = 8;                        // DP <= 256
#pragma unroll
    for (int which = 0; which < 2; ++which) {
      const Window<T> w = window(which);
      float f[kMax], ss = 0.0f;
#pragma unroll
      for (int i = 0; i < kMax; ++i) {
        const int d = lane + 32 * i;
        f[i] = d < a.D ? conv_silu<T>(w, a.taps_w[which], a.ntaps, item * a.D + d) : 0.0f;
        ss += f[i] * f[i];
      }
      float inv = 1.0f / sqrtf(warp_sum(ss) + 1e-6f);
      if (which == 0) inv *= 1.0f / sqrtf(static_cast<float>(a.D));
      float* out = (which == 0 ? a.q : a.k) + (static_cast<long long>(t) * a.G + item) * a.DP;
#pragma unroll
      for (int i = 0; i < kMax; ++i) {
        const int d = lane + 32 * i;
        if (d < a.DP) out[d] = f[i] * inv;
      }
    }
    return;
  }
  const int h = item - a.G;
  const Window<T> w = window(2);
  float* v = a.v + (static_cast<long long>(t) * a.N + h) * a.VP;
  for (int d = lane; d < a.VP; d += 32)
    v[d] = d < a.V ? conv_silu<T>(w, a.taps_w[2], a.ntaps, h * a.V + d) : 0.0f;
  float* g = a.g + (static_cast<long long>(t) * a.N + h) * a.DP;
  const float* z = a.z + t * a.ldz + h * a.D;
  const float rate = expf(a.a_log[h]);
  for (int d = lane; d < a.DP; d += 32)
    g[d] = d < a.D ? expf(-rate * softplus(z[d] + a.dt_bias[h * a.D + d])) : 0.0f;
  if (lane == 0)
    a.beta[static_cast<long long>(t) * a.N + h] = sigmoid(a.bz[t * a.ldb + h]);
}

// ---------------------------------------------------------------------------
struct MemoryIn {
  const void *q, *k, *v;     // [T, channels] views, row pitch ld
  const float *zi, *zf;      // [T, N] input and forget gate projections, row pitch ldg
  const float *ib, *fb;      // [N] biases
  float *qo, *ko;            // out: [T, N, DP]
  float* vo;                 // out: [T, N, VP]
  float *io, *fo;            // out: [T, N] log gates
  long long ld, ldg;
  int T, N, D, V, DP, VP;
  float cap, qscale;
};

__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

template <typename T>
__global__ void __launch_bounds__(256) memory_inputs_kernel(const MemoryIn a) {
  const long long t = blockIdx.x;
  const int nq = a.N * a.DP, nv = a.N * a.VP;
  const T* q = static_cast<const T*>(a.q) + t * a.ld;
  const T* k = static_cast<const T*>(a.k) + t * a.ld;
  const T* v = static_cast<const T*>(a.v) + t * a.ld;
  for (int e = threadIdx.x; e < nq; e += blockDim.x) {
    const int h = e / a.DP, d = e - h * a.DP;
    const bool in = d < a.D;
    a.qo[t * nq + e] = in ? to_f32<T>(q[h * a.D + d]) * a.qscale : 0.0f;
    a.ko[t * nq + e] = in ? to_f32<T>(k[h * a.D + d]) : 0.0f;
  }
  for (int e = threadIdx.x; e < nv; e += blockDim.x) {
    const int h = e / a.VP, d = e - h * a.VP;
    a.vo[t * nv + e] = d < a.V ? to_f32<T>(v[h * a.V + d]) : 0.0f;
  }
  for (int h = threadIdx.x; h < a.N; h += blockDim.x) {
    a.io[t * a.N + h] = soft_cap(a.zi[t * a.ldg + h] + a.ib[h], a.cap);
    a.fo[t * a.N + h] = -softplus(-soft_cap(a.zf[t * a.ldg + h] + a.fb[h], a.cap));
  }
}

// ---------------------------------------------------------------------------
constexpr int kChunk = 16;       // tokens staged at a time

struct ScanArgs {
  const float *q, *k;        // [T, G, DP]
  const float* g;            // delta: decays [T, N, DP]
  const float* v;            // [T, N, VP]
  const float *s0, *s1;      // delta: step sizes | memory: log input gate, log forget gate [T, N]
  float* out;                // [T, N, V]
  float* matrix;             // state, see the head of the file
  float* vector;
  float* scalar;
  const void* x[3];          // delta: convolution inputs of the step (q, k, v), row pitch ld
  void* taps;
  const long long* positions;
  const int* slots;
  const int* cu_q;
  long long ld;
  int G, N, D, V, VP, ntaps, num_slots, nd, np, cols;     // cols: value columns per CTA
  int elt;                   // bytes of an element of x and taps
};

// Convolution inputs of a portion's last tokens -> the slot's rows: the v channels of head h, and
// the q and k channels of its group from the group's first head.
template <typename T>
__device__ void keep_taps(const ScanArgs& a, const Portion& po, int slot, int h) {
  const int C = 2 * a.G * a.D + a.N * a.V;
  const int group = a.N / a.G, kvh = h / group;
  const long long last = a.positions[po.first] + po.count - 1;
  for (int o = 0; o < min(a.ntaps - 1, po.count); ++o) {
    const long long src = static_cast<long long>(po.first + po.count - 1 - o) * a.ld;
    T* dst = static_cast<T*>(a.taps) +
             (static_cast<long long>(slot) * a.ntaps + (last - o) % a.ntaps) * C;
    for (int d = threadIdx.x; d < a.V; d += blockDim.x)
      dst[2 * a.G * a.D + h * a.V + d] = static_cast<const T*>(a.x[2])[src + h * a.V + d];
    if (h % group == 0) {
      for (int d = threadIdx.x; d < a.D; d += blockDim.x) {
        dst[kvh * a.D + d] = static_cast<const T*>(a.x[0])[src + kvh * a.D + d];
        dst[(a.G + kvh) * a.D + d] = static_cast<const T*>(a.x[1])[src + kvh * a.D + d];
      }
    }
  }
}

template <int MODE, int RPL>
__host__ __device__ constexpr int stage_floats(int cols) {
  return kChunk * ((MODE == kDelta ? 3 : 2) * 8 * RPL + cols + 4);
}

template <int MODE, int RPL, int CPT>
__global__ void __launch_bounds__(256) recurrent_scan_kernel(const ScanArgs a) {
  constexpr int DP = 8 * RPL, P = RPL / 2;       // P: row pairs per lane
  constexpr int kRows = MODE == kDelta ? 3 : 2;  // staged rows of DP floats per token
  extern __shared__ float4 smem4[];
  float* smem = reinterpret_cast<float*>(smem4);
  const int stage = stage_floats<MODE, RPL>(a.cols);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int l = lane & 7;
  const int r = blockIdx.x, h = blockIdx.y, z = blockIdx.z;
  const int kvh = h / (a.N / a.G);
  const Portion po = portion_of(r, a.nd, a.cu_q);
  const int slot = a.slots[r];
  const int c_loc = (warp * 4 + (lane >> 3)) * CPT;      // first column of this lane, in the CTA's block
  const int c0 = z * a.cols + c_loc;
  if (slot < 0 || slot >= a.num_slots) {                 // padding of a captured batch
    for (int i = 0; i < po.count; ++i)
      for (int c = threadIdx.x; c < a.cols; c += blockDim.x)
        if (z * a.cols + c < a.V)
          a.out[(static_cast<long long>(po.first + i) * a.N + h) * a.V + z * a.cols + c] = 0.0f;
    return;
  }
  const bool fresh = a.positions[po.first] == 0;

  // tokens [i0, i0 + kChunk) of the portion -> stage b
  auto fetch = [&](int i0, int b) {
    float* s = smem + b * stage;
    const int n = min(kChunk, po.count - i0);
    constexpr int kVec = DP / 4;
    for (int e = threadIdx.x; e < n * kRows * kVec; e += blockDim.x) {
      const int i = e / (kRows * kVec), rem = e - i * (kRows * kVec);
      const int which = rem / kVec, d = (rem - which * kVec) * 4;
      const long long t = po.first + i0 + i;
      const float* src = which == 0 ? a.q + (t * a.G + kvh) * DP
                         : which == 1 ? a.k + (t * a.G + kvh) * DP
                                      : a.g + (t * a.N + h) * DP;
      copy16(s + (which * kChunk + i) * DP + d, src + d);
    }
    float* sv = s + kRows * kChunk * DP;
    const int vec = a.cols / 4;
    for (int e = threadIdx.x; e < n * vec; e += blockDim.x) {
      const int i = e / vec, c = (e - i * vec) * 4;
      const int col = z * a.cols + c;
      if (col < a.VP)
        copy16(sv + i * a.cols + c,
               a.v + (static_cast<long long>(po.first + i0 + i) * a.N + h) * a.VP + col);
      else
        *reinterpret_cast<float4*>(sv + i * a.cols + c) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float* ss = sv + kChunk * a.cols;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
      const long long at = static_cast<long long>(po.first + i0 + i) * a.N + h;
      copy4(ss + i, a.s0 + at);
      if (MODE == kMemory) copy4(ss + kChunk + i, a.s1 + at);
    }
  };

  fetch(0, 0);
  copy_commit();

  // state -> registers: lane l holds rows 4 (l + 8 i) .. + 3 of its columns
  uint64_t S[CPT][P], nv[MODE == kMemory ? P : 1];
  float m = 0.0f;
  const long long head_at = static_cast<long long>(slot) * a.N + h;
#pragma unroll
  for (int j = 0; j < CPT; ++j) {
    const bool in = !fresh && c0 + j < a.V;
    const float* src = a.matrix + (head_at * a.V + c0 + j) * DP + 4 * l;
#pragma unroll
    for (int i = 0; i < P / 2; ++i) {
      ulonglong2 u = make_ulonglong2(0, 0);
      if (in) u = *reinterpret_cast<const ulonglong2*>(src + 32 * i);
      S[j][2 * i] = u.x;
      S[j][2 * i + 1] = u.y;
    }
  }
  if (MODE == kMemory) {
#pragma unroll
    for (int i = 0; i < P / 2; ++i) {
      ulonglong2 u = make_ulonglong2(0, 0);
      if (!fresh)
        u = *reinterpret_cast<const ulonglong2*>(a.vector + head_at * DP + 4 * l + 32 * i);
      nv[2 * i] = u.x;
      nv[2 * i + 1] = u.y;
    }
    if (!fresh) m = a.scalar[head_at];
  }

  for (int i0 = 0; i0 < po.count; i0 += kChunk) {
    const int b = (i0 / kChunk) & 1;
    if (i0 + kChunk < po.count) fetch(i0 + kChunk, b ^ 1);
    copy_commit();
    copy_wait<1>();
    __syncthreads();
    const int n = min(kChunk, po.count - i0);
    const float* sq = smem + b * stage;
    const float* sk = sq + kChunk * DP;
    const float* sg = sk + kChunk * DP;                         // delta only
    const float* sv = sq + kRows * kChunk * DP;
    const float* ss = sv + kChunk * a.cols;

    // matrix memory: running maximum and the two factors of every token of the chunk, lane t
    // computing token t's
    float keep = 0.0f, add = 0.0f, floor_den = 0.0f;
    if (MODE == kMemory) {
      float f = 0.0f, F = 0.0f, M = -INFINITY, ig = -INFINITY;
      if (lane < n) {
        ig = M = ss[lane];
        f = F = ss[kChunk + lane];
      }
#pragma unroll
      for (int d = 1; d < kChunk; d <<= 1) {
        const float Fp = __shfl_up_sync(0xffffffffu, F, d);
        const float Mp = __shfl_up_sync(0xffffffffu, M, d);
        if (lane >= d) {
          M = fmaxf(M, Mp + F);
          F += Fp;
        }
      }
      const float mt = fmaxf(m + F, M);
      float before = __shfl_up_sync(0xffffffffu, mt, 1);
      if (lane == 0) before = m;
      keep = expf(f + (before - mt));        // the difference of the maxima is (nearly) exact
      add = expf(ig - mt);
      floor_den = expf(-mt);
      m = __shfl_sync(0xffffffffu, mt, n - 1);
    }

    for (int i = 0; i < n; ++i) {
      uint64_t kk[P], qq[P];
#pragma unroll
      for (int u = 0; u < P / 2; ++u) {
        const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(sk + i * DP + 4 * l + 32 * u);
        const ulonglong2 y = *reinterpret_cast<const ulonglong2*>(sq + i * DP + 4 * l + 32 * u);
        kk[2 * u] = x.x; kk[2 * u + 1] = x.y;
        qq[2 * u] = y.x; qq[2 * u + 1] = y.y;
      }
      float v[CPT], o[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) v[j] = sv[i * a.cols + c_loc + j];
      if (MODE == kDelta) {
        const float beta = ss[i];
        uint64_t d0[CPT], d1[CPT];
#pragma unroll
        for (int j = 0; j < CPT; ++j) d0[j] = d1[j] = 0;
#pragma unroll
        for (int u = 0; u < P / 2; ++u) {
          const ulonglong2 g = *reinterpret_cast<const ulonglong2*>(sg + i * DP + 4 * l + 32 * u);
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            S[j][2 * u] = mul2(S[j][2 * u], g.x);
            S[j][2 * u + 1] = mul2(S[j][2 * u + 1], g.y);
            d0[j] = fma2(S[j][2 * u], kk[2 * u], d0[j]);
            d1[j] = fma2(S[j][2 * u + 1], kk[2 * u + 1], d1[j]);
          }
        }
        float d[CPT];
#pragma unroll
        for (int j = 0; j < CPT; ++j) d[j] = halves_sum(d0[j]) + halves_sum(d1[j]);
#pragma unroll
        for (int w = 1; w < 8; w <<= 1) {
#pragma unroll
          for (int j = 0; j < CPT; ++j) d[j] += __shfl_xor_sync(0xffffffffu, d[j], w);
        }
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          const uint64_t u2 = both(beta * (v[j] - d[j]));
          uint64_t e0 = 0, e1 = 0;
#pragma unroll
          for (int u = 0; u < P; u += 2) {
            S[j][u] = fma2(kk[u], u2, S[j][u]);
            S[j][u + 1] = fma2(kk[u + 1], u2, S[j][u + 1]);
            e0 = fma2(S[j][u], qq[u], e0);
            e1 = fma2(S[j][u + 1], qq[u + 1], e1);
          }
          o[j] = halves_sum(e0) + halves_sum(e1);
        }
#pragma unroll
        for (int w = 1; w < 8; w <<= 1) {
#pragma unroll
          for (int j = 0; j < CPT; ++j) o[j] += __shfl_xor_sync(0xffffffffu, o[j], w);
        }
      } else {
        const uint64_t a2 = both(__shfl_sync(0xffffffffu, keep, i));
        const uint64_t b2 = both(__shfl_sync(0xffffffffu, add, i));
        const float low = __shfl_sync(0xffffffffu, floor_den, i);
        uint64_t e = 0;
#pragma unroll
        for (int u = 0; u < P; ++u) {
          kk[u] = mul2(kk[u], b2);
          nv[u] = fma2(nv[u], a2, kk[u]);
          e = fma2(nv[u], qq[u], e);
        }
        float den = halves_sum(e);
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          const uint64_t v2 = both(v[j]);
          uint64_t e0 = 0, e1 = 0;
#pragma unroll
          for (int u = 0; u < P; u += 2) {
            S[j][u] = fma2(kk[u], v2, mul2(S[j][u], a2));
            S[j][u + 1] = fma2(kk[u + 1], v2, mul2(S[j][u + 1], a2));
            e0 = fma2(S[j][u], qq[u], e0);
            e1 = fma2(S[j][u + 1], qq[u + 1], e1);
          }
          o[j] = halves_sum(e0) + halves_sum(e1);
        }
#pragma unroll
        for (int w = 1; w < 8; w <<= 1) {
          den += __shfl_xor_sync(0xffffffffu, den, w);
#pragma unroll
          for (int j = 0; j < CPT; ++j) o[j] += __shfl_xor_sync(0xffffffffu, o[j], w);
        }
        den = fmaxf(fabsf(den), low) + 1e-6f;
#pragma unroll
        for (int j = 0; j < CPT; ++j) o[j] /= den;
      }
      float* dst = a.out + (static_cast<long long>(po.first + i0 + i) * a.N + h) * a.V + c0;
      if (l == 0) {
#pragma unroll
        for (int j = 0; j < CPT; ++j)
          if (c0 + j < a.V) dst[j] = o[j];
      }
    }
    __syncthreads();           // stage b is refilled next
  }

  // registers -> state
#pragma unroll
  for (int j = 0; j < CPT; ++j) {
    if (c0 + j >= a.V) continue;
    float* dst = a.matrix + (head_at * a.V + c0 + j) * DP + 4 * l;
#pragma unroll
    for (int i = 0; i < P / 2; ++i)
      *reinterpret_cast<ulonglong2*>(dst + 32 * i) = make_ulonglong2(S[j][2 * i], S[j][2 * i + 1]);
  }
  if (MODE == kMemory) {
    if (z == 0 && threadIdx.x < 8) {
#pragma unroll
      for (int i = 0; i < P / 2; ++i)
        *reinterpret_cast<ulonglong2*>(a.vector + head_at * DP + 4 * l + 32 * i) =
            make_ulonglong2(nv[2 * i], nv[2 * i + 1]);
      if (threadIdx.x == 0) a.scalar[head_at] = m;
    }
  } else if (z == 0 && a.ntaps > 1) {
    if (a.elt == 2) keep_taps<uint16_t>(a, po, slot, h);
    else keep_taps<uint32_t>(a, po, slot, h);
  }
}

template <int MODE, int RPL, int CPT>
static int launch_scan(const ScanArgs& a, int requests, cudaStream_t s) {
  const int smem = 2 * stage_floats<MODE, RPL>(a.cols) * static_cast<int>(sizeof(float));
  static bool done[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -9;
  if (!done[dev]) {
    cudaError_t e = cudaFuncSetAttribute(recurrent_scan_kernel<MODE, RPL, CPT>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    done[dev] = true;
  }
  dim3 grid(requests, a.N, (a.V + a.cols - 1) / a.cols);
  recurrent_scan_kernel<MODE, RPL, CPT><<<grid, a.cols / CPT * 8, smem, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

// Columns per CTA: as many as leave two CTAs for every SM.
static int scan_columns(int V, int ctas_per_block, int most) {
  int cols = 16;
  while (cols < most && cols < V) cols *= 2;
  while (cols > 16 && static_cast<long long>(ctas_per_block) * ((V + cols - 1) / cols) <
                          2ll * sm_count())
    cols /= 2;
  return cols;
}

template <int MODE, int RPL>
static int dispatch_scan(ScanArgs& a, int requests, cudaStream_t s) {
  a.cols = scan_columns(a.V, requests * a.N, RPL > 16 ? 64 : 128);
  if constexpr (RPL <= 16) {
    if (a.cols >= 64) return launch_scan<MODE, RPL, 4>(a, requests, s);
  }
  if (a.cols >= 32) return launch_scan<MODE, RPL, 2>(a, requests, s);
  return launch_scan<MODE, RPL, 1>(a, requests, s);
}

template <int MODE>
static int dispatch_scan(ScanArgs& a, int DP, int requests, cudaStream_t s) {
  switch (DP) {
    case 32: return dispatch_scan<MODE, 4>(a, requests, s);
    case 64: return dispatch_scan<MODE, 8>(a, requests, s);
    case 96: return dispatch_scan<MODE, 12>(a, requests, s);
    case 128: return dispatch_scan<MODE, 16>(a, requests, s);
    case 192: return dispatch_scan<MODE, 24>(a, requests, s);
    case 256: return dispatch_scan<MODE, 32>(a, requests, s);
  }
  return -20;
}

// ---------------------------------------------------------------------------
struct HeadNormArgs {
  const float* o;            // [T, N, V]
  const float* w;            // norm weight: [V] shared by the heads, or [N * V]
  const void* z;             // [T, N * V] gate projection, row pitch ldz
  void* out;                 // [T, N * V], row pitch ldo
  long long ldz, ldo;
  int T, N, V, per_head;
  float eps, scale;
};

template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const HeadNormArgs a) {
  const int lane = threadIdx.x & 31;
  const long long row = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (row >= static_cast<long long>(a.T) * a.N) return;
  const long long t = row / a.N;
  const int h = static_cast<int>(row - t * a.N);
  const float* o = a.o + row * a.V;
  float ss = 0.0f;
  for (int c = lane; c < a.V; c += 32) ss += o[c] * o[c];
  const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(a.V) + a.eps) * a.scale;
  const float* w = a.w + (a.per_head ? h * a.V : 0);
  const T* z = static_cast<const T*>(a.z) + t * a.ldz + h * a.V;
  T* out = static_cast<T*>(a.out) + t * a.ldo + h * a.V;
  for (int c = lane; c < a.V; c += 32)
    out[c] = from_f32<T>(o[c] * inv * w[c] * sigmoid(to_f32<T>(z[c])));
}

}  // namespace recurrent
}  // namespace b200

using namespace b200;
using namespace b200::recurrent;

// Padded key rows of a head dimension (-20: larger than the scan covers).
B200_API int b200_recurrent_rows(int D) {
  const int sizes[] = {32, 64, 96, 128, 192, 256};
  for (int n : sizes)
    if (D <= n) return n;
  return -20;
}

// Convolution + SiLU, unit vectors, decays and step sizes of every token of the step.  dtype (of
// q, k, v projections and taps): 0 bf16, 2 fp32.
B200_API int b200_delta_inputs(const void* xq, const void* xk, const void* xv, long long ld,
                               const float* wq, const float* wk, const float* wv, int ntaps,
                               const void* taps, int num_slots, const float* z, long long ldz,
                               const float* bz, long long ldb, const float* dt_bias,
                               const float* a_log, float* q, float* k, float* g, float* v,
                               float* beta, const long long* positions, const int* slots,
                               const int* cu_q, int T, int G, int N, int D, int V, int DP, int VP,
                               int nd, int np, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (G <= 0 || N <= 0 || N % G != 0 || D <= 0 || D > DP || DP > 256 || V <= 0 || V > VP ||
      ntaps < 1 || ntaps > kMaxTaps || (dtype != 0 && dtype != 2))
    return -2;
  DeltaIn a;
  a.x[0] = xq; a.x[1] = xk; a.x[2] = xv; a.taps_w[0] = wq; a.taps_w[1] = wk; a.taps_w[2] = wv;
  a.taps = taps; a.z = z; a.bz = bz; a.dt_bias = dt_bias; a.a_log = a_log; a.q = q; a.k = k;
  a.g = g; a.v = v; a.beta = beta; a.positions = positions; a.slots = slots; a.cu_q = cu_q;
  a.ld = ld; a.ldz = ldz; a.ldb = ldb; a.T = T; a.G = G; a.N = N; a.D = D; a.V = V; a.DP = DP;
  a.VP = VP; a.ntaps = ntaps; a.num_slots = num_slots; a.nd = nd; a.np = np;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  dim3 grid(T, (G + N + 7) / 8);
  if (dtype == 0) delta_inputs_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(a);
  else delta_inputs_kernel<float><<<grid, 256, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

// fp32 inputs and log gates of the matrix memory.  dtype (of q, k, v): 0 bf16, 2 fp32.
B200_API int b200_memory_inputs(const void* q, const void* k, const void* v, long long ld,
                                const float* zi, const float* zf, long long ldg, const float* ib,
                                const float* fb, float cap, float qscale, float* qo, float* ko, float* vo,
                                float* io, float* fo, int T, int N, int D, int V, int DP, int VP,
                                int dtype, void* stream) {
  if (T <= 0) return 0;
  if (N <= 0 || D <= 0 || D > DP || V <= 0 || V > VP || (dtype != 0 && dtype != 2)) return -2;
  MemoryIn a;
  a.q = q; a.k = k; a.v = v; a.zi = zi; a.zf = zf; a.ib = ib; a.fb = fb; a.qo = qo; a.ko = ko; a.vo = vo;
  a.io = io; a.fo = fo; a.ld = ld; a.ldg = ldg; a.T = T; a.N = N; a.D = D; a.V = V; a.DP = DP;
  a.VP = VP; a.cap = cap; a.qscale = qscale;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 0) memory_inputs_kernel<__nv_bfloat16><<<T, 256, 0, s>>>(a);
  else memory_inputs_kernel<float><<<T, 256, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

// Gated delta rule over the portions of a step (nd single tokens, then np portions by cu_q).
B200_API int b200_delta_scan(const float* q, const float* k, const float* g, const float* v,
                             const float* beta, float* out, float* matrix, const void* xq,
                             const void* xk, const void* xv, long long ld, void* taps, int ntaps,
                             const long long* positions, const int* slots, int num_slots,
                             const int* cu_q, int G, int N, int D, int V, int DP, int VP, int nd,
                             int np, int elt, void* stream) {
  if (nd + np <= 0) return 0;
  if (G <= 0 || N <= 0 || N % G != 0 || (VP % 4) != 0 || ntaps < 1 || (elt != 2 && elt != 4))
    return -2;
  ScanArgs a{};
  a.q = q; a.k = k; a.g = g; a.v = v; a.s0 = beta; a.out = out; a.matrix = matrix;
  a.x[0] = xq; a.x[1] = xk; a.x[2] = xv; a.ld = ld; a.taps = taps; a.ntaps = ntaps;
  a.positions = positions; a.slots = slots; a.num_slots = num_slots; a.cu_q = cu_q; a.G = G;
  a.N = N; a.D = D; a.V = V; a.VP = VP; a.nd = nd; a.np = np; a.elt = elt;
  return dispatch_scan<kDelta>(a, DP, nd + np, static_cast<cudaStream_t>(stream));
}

// Matrix memory over the portions of a step; the state is (matrix, vector n, scalar m).
B200_API int b200_memory_scan(const float* q, const float* k, const float* v, const float* li,
                              const float* lf, float* out, float* matrix, float* vector,
                              float* scalar, const long long* positions, const int* slots,
                              int num_slots, const int* cu_q, int N, int D, int V, int DP, int VP,
                              int nd, int np, void* stream) {
  if (nd + np <= 0) return 0;
  if (N <= 0 || (VP % 4) != 0) return -2;
  ScanArgs a{};
  a.q = q; a.k = k; a.v = v; a.s0 = li; a.s1 = lf; a.out = out; a.matrix = matrix;
  a.vector = vector; a.scalar = scalar; a.positions = positions; a.slots = slots;
  a.num_slots = num_slots; a.cu_q = cu_q; a.G = N; a.N = N; a.D = D; a.V = V; a.VP = VP; a.nd = nd;
  a.np = np; a.ntaps = 1;
  return dispatch_scan<kMemory>(a, DP, nd + np, static_cast<cudaStream_t>(stream));
}

// out = o / rms(o) per head * w * sigmoid(z) * scale.  per_head: w is [N * V], else [V].  dtype (of
// z and out): 0 bf16, 2 fp32.
B200_API int b200_head_norm_gate(const float* o, const float* w, int per_head, const void* z,
                                 long long ldz, void* out, long long ldo, float eps, float scale,
                                 int T, int N, int V, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (N <= 0 || V <= 0 || (dtype != 0 && dtype != 2)) return -2;
  HeadNormArgs a;
  a.o = o; a.w = w; a.z = z; a.out = out; a.ldz = ldz; a.ldo = ldo; a.T = T; a.N = N; a.V = V;
  a.per_head = per_head; a.eps = eps; a.scale = scale;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const long long blocks = (static_cast<long long>(T) * N + 7) / 8;
  if (dtype == 0) head_norm_gate_kernel<__nv_bfloat16><<<static_cast<int>(blocks), 256, 0, s>>>(a);
  else head_norm_gate_kernel<float><<<static_cast<int>(blocks), 256, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}
