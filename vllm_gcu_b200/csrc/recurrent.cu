// Linear recurrences with a matrix state per head (sm_100a): gated delta rule with one decay per
// key channel, the matrix memory with exponential gates (mLSTM), and time mixing of the RWKV kind
// (one decay per key channel, a bonus for the current token):
//   o_t = S^T r_t + (r_t . (u k_t)) v_t,  then  S = diag(w_t) S + k_t v_t^T
//
//   delta_inputs    short causal convolution + SiLU of q, k, v, unit vectors, decays, step sizes
//   memory_inputs   q (scaled), k, v in fp32, log gates of the matrix memory
//   wkv_inputs      r, k, v in fp32, decays and the bonus' products r . (u k)
//   recurrent_scan  the recurrence over portions of prompts
//   head_norm_gate  o / rms(o) per head, times the norm weight, a sigmoid or SiLU gate and a factor
//   recurrent_step  all of these (and the narrow projections in front of them) for requests that
//                   bring a single token: one CTA per request and head
//
// State of a request, addressed by its state slot, fp32 throughout:
//   matrix  [slot, head, vdim, DP]      S transposed: a value column's key entries are contiguous
//   vector  [slot, head, DP], scalar [slot, head]      (matrix memory: normaliser n, maximum m)
//   taps    [slot, taps, channels] in the model's type: row p % taps holds the convolution input
//           of position p.  A step reads the rows of positions in front of its portion before
//           the scan overwrites them; a single token writes a row that no one reads in its step.
// A portion that starts at position 0 starts from zeros whatever the slot holds, so slots need no
// clearing.  DP is the head dimension rounded up (b200_recurrent_rows); the padding stays zero.
//
// The scan splits a head's value columns over threads: they are independent of each other.  LPC
// lanes share a column (RPL key rows each, in registers), CPT columns per lane group; a CTA holds a
// block of columns of one head of one request and walks its tokens in order, inputs staged through
// shared memory by cp.async one chunk ahead.  Two lanes per column keep the arithmetic units busy
// when there are heads enough for every scheduler; eight shorten the chain from token to token when
// there are few.  The normaliser of the matrix memory is one more column whose value is always 1.
// The result of a token does not depend on where the prompt was cut.
#include "common.cuh"

namespace b200 {
namespace recurrent {

constexpr int kDelta = 0, kMemory = 1, kWkv = 2;

// fp32 pairs: two multiply-adds per instruction
struct __align__(16) Quad {
  float2 x, y;
};
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) { return __ffma2_rn(a, b, c); }
__device__ __forceinline__ float2 mul2(float2 a, float2 b) { return __fmul2_rn(a, b); }
__device__ __forceinline__ float2 both(float x) { return make_float2(x, x); }
__device__ __forceinline__ float halves_sum(float2 x) { return x.x + x.y; }

__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) {
  return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)));
}
// fp32 forms for 16-bit models: the fast exponential and division, relative errors near 1e-6; the
// logarithm of 1 + e switches to its series where e would be rounded away
template <typename T>
__device__ __forceinline__ float sigmoid_t(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.0f, 1.0f + __expf(-z));
  else return sigmoid(z);
}
template <typename T>
__device__ __forceinline__ float softplus_t(float z) {
  if constexpr (sizeof(T) == 2) {
    const float e = __expf(-fabsf(z));
    const float l = e < 0.02f ? fmaf(e * e, fmaf(e, 1.0f / 3.0f, -0.5f), e) : __logf(1.0f + e);
    return fmaxf(z, 0.0f) + l;
  } else {
    return softplus(z);
  }
}
template <typename T>
__device__ __forceinline__ float inv_root(float z) {
  if constexpr (sizeof(T) == 2) return rsqrtf(z);
  else return 1.0f / sqrtf(z);
}
template <typename T>
__device__ __forceinline__ float exp_t(float z) {
  if constexpr (sizeof(T) == 2) return __expf(z);
  else return expf(z);
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
  const float* taps_w[3];    // [taps, channels] convolution weights, last row: current token
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

constexpr int kMaxTaps = 8;
constexpr int kStrip = 8;        // tokens one warp walks

template <typename T, int V>
__device__ __forceinline__ void load_n(const T* p, float (&f)[V]) {
  if constexpr (V == 4 && sizeof(T) == 2) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else if constexpr (V == 4) {
    const float4 u = *reinterpret_cast<const float4*>(p);
    f[0] = u.x; f[1] = u.y; f[2] = u.z; f[3] = u.w;
  } else {
    f[0] = to_f32<T>(p[0]);
  }
}
// V elements as they lie in memory
template <typename T, int V>
struct Raw {
  T e;
};
template <>
struct Raw<__nv_bfloat16, 4> {
  uint2 e;
};
template <>
struct Raw<float, 4> {
  float4 e;
};
template <typename T, int V>
__device__ __forceinline__ void unpack_raw(const Raw<T, V>& r, float (&f)[V]) {
  if constexpr (V == 4 && sizeof(T) == 2) {
    const float2 a = unpack_bf16x2(r.e.x), b = unpack_bf16x2(r.e.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else if constexpr (V == 4) {
    f[0] = r.e.x; f[1] = r.e.y; f[2] = r.e.z; f[3] = r.e.w;
  } else {
    f[0] = to_f32<T>(r.e);
  }
}
template <int V>
__device__ __forceinline__ void store_n(float* p, const float (&f)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else p[0] = f[0];
}
// SiLU at the precision of the model's type
template <typename T>
__device__ __forceinline__ float silu(float x) {
  if constexpr (sizeof(T) == 2) return __fdividef(x, 1.0f + __expf(-x));
  else return x / (1.0f + expf(-x));
}

// A CTA: kStrip tokens; every warp walks its items, V neighbouring channels per lane (32 V channels
// at a time).  Items: [0, G) q heads, [G, 2G) k heads, [2G, 2G + N) v heads, [2G + N, 2G + 2N)
// decays.
template <typename T, int NT, int V>
__global__ void __launch_bounds__(256, 2) delta_inputs_kernel(const DeltaIn a) {
  __shared__ int s_first[kStrip], s_slot[kStrip];   // portion's first token (-1: none), its slot
  __shared__ long long s_pos[kStrip];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * kStrip;
  const int t1 = min(t0 + kStrip, a.T);
  if (threadIdx.x < kStrip) {
    const int t = t0 + threadIdx.x;
    s_first[threadIdx.x] = -1;
    if (t < t1) {
      const TokenPlace pl = token_place(t, a.nd, a.np, a.cu_q);
      if (pl.req >= 0) {
        s_first[threadIdx.x] = portion_of(pl.req, a.nd, a.cu_q).first;
        s_slot[threadIdx.x] = a.slots[pl.req];
        s_pos[threadIdx.x] = a.positions[t];
      }
    }
  }
  __syncthreads();
  const int C = 2 * a.G * a.D + a.N * a.V;
  const float qscale = 1.0f / sqrtf(static_cast<float>(a.D));
  for (int item = blockIdx.y * 8 + warp; item < 2 * a.G + 2 * a.N; item += gridDim.y * 8) {
    if (item >= 2 * a.G + a.N) {                   // decays and step sizes
      const int h = item - 2 * a.G - a.N;
      const float rate = expf(a.a_log[h]);
      for (int d = lane * V; d < a.DP; d += 32 * V) {
        float bias[V];
#pragma unroll
        for (int i = 0; i < V; ++i) bias[i] = d + i < a.D ? a.dt_bias[h * a.D + d + i] : 0.0f;
        float g[kStrip][V];                        // all rows of the strip in flight at once
#pragma unroll
        for (int u = 0; u < kStrip; ++u) {
#pragma unroll
          for (int i = 0; i < V; ++i) g[u][i] = 0.0f;
          if (d < a.D && t0 + u < t1) load_n<float, V>(a.z + (t0 + u) * a.ldz + h * a.D + d, g[u]);
        }
#pragma unroll
        for (int u = 0; u < kStrip; ++u) {
          if (t0 + u >= t1) break;
#pragma unroll
          for (int i = 0; i < V; ++i)
            g[u][i] = d < a.D ? exp_t<T>(-rate * softplus_t<T>(g[u][i] + bias[i])) : 0.0f;
          store_n<V>(a.g + (static_cast<long long>(t0 + u) * a.N + h) * a.DP + d, g[u]);
        }
      }
      for (int t = t0 + lane; t < t1; t += 32)
        a.beta[static_cast<long long>(t) * a.N + h] = sigmoid(a.bz[t * a.ldb + h]);
      continue;
    }
    const int which = item < a.G ? 0 : item < 2 * a.G ? 1 : 2;
    const int head = which == 0 ? item : which == 1 ? item - a.G : item - 2 * a.G;
    const int dim = which == 2 ? a.V : a.D, pitch = which == 2 ? a.VP : a.DP;
    const int ring_off = (which == 0 ? 0 : which == 1 ? a.G * a.D : 2 * a.G * a.D) + head * dim;
    const T* x = static_cast<const T*>(a.x[which]) + head * dim;
    const float* wt = a.taps_w[which] + head * dim;
    const int wld = (which == 2 ? a.N : a.G) * dim;
    float* out = (which == 0 ? a.q : which == 1 ? a.k : a.v) + head * pitch;
    const long long ldo = static_cast<long long>(which == 2 ? a.N : a.G) * pitch;
    const int passes = (pitch + 32 * V - 1) / (32 * V);
    float inv_sum[kStrip];
    // q and k of more channels than one pass holds: a first walk over all passes for the norms
    const bool unit = which < 2;
    for (int walk = unit && passes > 1 ? 0 : 1; walk < 2; ++walk) {
      for (int ps = 0; ps < passes; ++ps) {
        const int d = (ps * 32 + lane) * V;
        const bool in = d < dim;
        Raw<T, V> rows[kStrip];                    // all rows of the strip in flight at once
#pragma unroll
        for (int u = 0; u < kStrip; ++u) {
          rows[u] = Raw<T, V>{};
          if (in && t0 + u < t1)
            rows[u] = *reinterpret_cast<const Raw<T, V>*>(
                x + static_cast<long long>(t0 + u) * a.ld + d);
        }
        float w[NT][V];                            // [o]: tap that meets the input of o tokens ago
#pragma unroll
        for (int o = 0; o < NT; ++o) {
#pragma unroll
          for (int i = 0; i < V; ++i) w[o][i] = 0.0f;
          if (in && o < a.ntaps) load_n<float, V>(wt + (a.ntaps - 1 - o) * wld + d, w[o]);
        }
        float past[NT][V];                         // [o]: input of o tokens ago
#pragma unroll
        for (int o = 0; o < NT; ++o) {
#pragma unroll
          for (int i = 0; i < V; ++i) past[o][i] = 0.0f;
        }
#pragma unroll
        for (int u = 0; u < kStrip; ++u) {
          const int t = t0 + u;
          const int first = s_first[u];
          if (t >= t1 || first < 0) break;         // (padding rows end the step)
          if (u == 0 || t == first) {              // the inputs in front of the walk
            const long long pos = s_pos[u];
            const int slot = s_slot[u];
#pragma unroll
            for (int o = 1; o < NT; ++o) {
#pragma unroll
              for (int i = 0; i < V; ++i) past[o - 1][i] = 0.0f;
              if (!in || o >= a.ntaps || pos - o < 0) continue;
              if (t - o >= first) {
                load_n<T, V>(x + static_cast<long long>(t - o) * a.ld + d, past[o - 1]);
              } else if (slot >= 0 && slot < a.num_slots) {
                load_n<T, V>(static_cast<const T*>(a.taps) +
                                 (static_cast<long long>(slot) * a.ntaps + (pos - o) % a.ntaps) * C +
                                 ring_off + d, past[o - 1]);
              }
            }
          }
#pragma unroll
          for (int o = NT - 1; o > 0; --o) {
#pragma unroll
            for (int i = 0; i < V; ++i) past[o][i] = past[o - 1][i];
          }
          unpack_raw<T, V>(rows[u], past[0]);
          float f[V], ss = 0.0f;
          if constexpr (V == 4) {
            float2 c0 = both(0.0f), c1 = both(0.0f);
#pragma unroll
            for (int o = NT - 1; o >= 0; --o) {
              c0 = fma2(make_float2(w[o][0], w[o][1]), make_float2(past[o][0], past[o][1]), c0);
              c1 = fma2(make_float2(w[o][2], w[o][3]), make_float2(past[o][2], past[o][3]), c1);
            }
            f[0] = c0.x; f[1] = c0.y; f[2] = c1.x; f[3] = c1.y;
          } else {
            f[0] = 0.0f;
#pragma unroll
            for (int o = NT - 1; o >= 0; --o) f[0] += w[o][0] * past[o][0];
          }
#pragma unroll
          for (int i = 0; i < V; ++i) {
            f[i] = silu<T>(f[i]);
            ss += f[i] * f[i];
          }
          if (unit) {
            float inv;
            if (passes == 1) {
              inv = inv_root<T>(warp_sum(ss) + 1e-6f);
            } else if (walk == 0) {
              const float sum = warp_sum(ss);
              inv_sum[u] = ps == 0 ? sum : inv_sum[u] + sum;
              continue;
            } else {
              inv = inv_root<T>(inv_sum[u] + 1e-6f);
            }
            if (which == 0) inv *= qscale;
#pragma unroll
            for (int i = 0; i < V; ++i) f[i] *= inv;
          }
          if (d < pitch) store_n<V>(out + t * ldo + d, f);
        }
      }
    }
  }
}

// ---------------------------------------------------------------------------
struct MemoryIn {
  const void *q, *k, *v;     // [T, channels] views, row pitch ld
  const float *zi, *zf;      // [T, N] input and forget gate projections, row pitch ldg
  const float *ib, *fb;      // [N] biases
  const float* scalar;       // state m [slots, N]
  float *qo, *ko;            // out: [T, N, DP]
  float* vo;                 // out: [T, N, VP], column V: 1
  float *io, *fo;            // out: [T, N] log gates
  float* m0;                 // out: [requests, N] m in front of the portion
  const long long* positions;
  const int* slots;
  const int* cu_q;
  long long ld, ldg;
  int T, N, D, V, DP, VP, num_slots, nd, np;
  float cap, qscale;
};

__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

template <typename T, int W>
__global__ void __launch_bounds__(256) memory_inputs_kernel(const MemoryIn a) {
  const long long t = blockIdx.x;
  const int kd = a.DP / W, kv = a.VP / W;
  const int nq = a.N * kd, nv = a.N * kv;
  for (int e = threadIdx.x; e < 2 * nq + nv; e += blockDim.x) {
    const int which = e < nq ? 0 : e < 2 * nq ? 1 : 2;
    const int r = which == 0 ? e : which == 1 ? e - nq : e - 2 * nq;
    const int per = which == 2 ? kv : kd, dim = which == 2 ? a.V : a.D;
    const int h = r / per, d = (r - h * per) * W;
    const T* x = static_cast<const T*>(which == 0 ? a.q : which == 1 ? a.k : a.v) + t * a.ld +
                 h * dim;
    float f[W];
#pragma unroll
    for (int i = 0; i < W; ++i) f[i] = 0.0f;
    if (d < dim) load_n<T, W>(x + d, f);
    if (which == 0) {
#pragma unroll
      for (int i = 0; i < W; ++i) f[i] *= a.qscale;
    }
    if (which == 2) {
#pragma unroll
      for (int i = 0; i < W; ++i)
        if (d + i == a.V) f[i] = 1.0f;
    }
    float* out = which == 0 ? a.qo : which == 1 ? a.ko : a.vo;
    store_n<W>(out + (t * a.N + h) * (which == 2 ? a.VP : a.DP) + d, f);
  }
  const TokenPlace pl = token_place(static_cast<int>(t), a.nd, a.np, a.cu_q);
  for (int h = threadIdx.x; h < a.N; h += blockDim.x) {
    a.io[t * a.N + h] = soft_cap(a.zi[t * a.ldg + h] + a.ib[h], a.cap);
    a.fo[t * a.N + h] = -softplus(-soft_cap(a.zf[t * a.ldg + h] + a.fb[h], a.cap));
    if (pl.req >= 0 && pl.first) {
      const int slot = a.slots[pl.req];
      a.m0[static_cast<long long>(pl.req) * a.N + h] =
          a.positions[t] == 0 || slot < 0 || slot >= a.num_slots
              ? 0.0f : a.scalar[static_cast<long long>(slot) * a.N + h];
    }
  }
}

// ---------------------------------------------------------------------------
struct WkvIn {
  const void *r, *k, *v;     // [T, N * D] views, row pitch ld
  const float* z;            // [T, N * D] decay projection
  const float *base, *bonus; // [N * D]
  float *ro, *ko, *go;       // out: [T, N, DP]
  float* vo;                 // out: [T, N, VP]
  float* now;                // out: [T, N] r . (bonus k)
  long long ld, ldz;
  int T, N, D, DP, VP;
};

// LPH lanes per token and head, W neighbouring channels each.
template <typename T, int W, int LPH>
__global__ void __launch_bounds__(256) wkv_inputs_kernel(const WkvIn a) {
  const long long job = (blockIdx.x * 256ll + threadIdx.x) / LPH;
  if (job >= static_cast<long long>(a.T) * a.N) return;      // (whole groups of lanes leave)
  const int l = threadIdx.x & (LPH - 1);
  const long long t = job / a.N;
  const int h = static_cast<int>(job - t * a.N), at = h * a.D;
  const long long row = t * a.ld + at;
  float sum = 0.0f;
  for (int d = l * W; d < a.DP; d += LPH * W) {
    float r[W], k[W], v[W], g[W];
#pragma unroll
    for (int i = 0; i < W; ++i) r[i] = k[i] = v[i] = g[i] = 0.0f;
    if (d < a.D) {
      float b[W], u[W];
      load_n<T, W>(static_cast<const T*>(a.r) + row + d, r);
      load_n<T, W>(static_cast<const T*>(a.k) + row + d, k);
      load_n<T, W>(static_cast<const T*>(a.v) + row + d, v);
      load_n<float, W>(a.z + t * a.ldz + at + d, g);
      load_n<float, W>(a.base + at + d, b);
      load_n<float, W>(a.bonus + at + d, u);
#pragma unroll
      for (int i = 0; i < W; ++i) {
        g[i] = exp_t<T>(-exp_t<T>(g[i] + b[i]));
        sum += r[i] * u[i] * k[i];
      }
    }
    store_n<W>(a.ro + job * a.DP + d, r);
    store_n<W>(a.ko + job * a.DP + d, k);
    store_n<W>(a.go + job * a.DP + d, g);
    if (d < a.VP) store_n<W>(a.vo + job * a.VP + d, v);
  }
  const unsigned int mask = LPH == 32 ? 0xffffffffu
                                      : ((1u << (LPH & 31)) - 1u) << (threadIdx.x & (32 - LPH));
#pragma unroll
  for (int o = 1; o < LPH; o <<= 1) sum += __shfl_xor_sync(mask, sum, o);
  if (l == 0) a.now[job] = sum;
}

template <typename T>
__global__ void __launch_bounds__(256) tanh_rows_kernel(const float* x, T* out, long long n) {
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i < n) out[i] = from_f32<T>(tanhf(x[i]));
}

// ---------------------------------------------------------------------------
constexpr int kChunk = 16;       // tokens staged at a time

struct ScanArgs {
  const float *q, *k;        // [T, G, DP]
  const float* g;            // delta, wkv: decays [T, N, DP]
  const float* v;            // [T, N, VP]
  const float *s0, *s1;      // delta: step sizes | memory: log input gate, log forget gate |
                             // wkv: products of the bonus [T, N]
  float* out;                // [T, N, V] (memory: not yet divided)
  float *nq, *low;           // memory: [T, N] normaliser . q, exp(-m)
  const float* m0;           // memory: [requests, N] m in front of the portion
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

template <int MODE, int DP>
__host__ __device__ constexpr int stage_floats(int cols) {
  return kChunk * ((MODE == kMemory ? 2 : 3) * DP + cols + 4);
}

template <int MODE, int LPC, int RPL, int CPT>
__global__ void __launch_bounds__(128) recurrent_scan_kernel(const ScanArgs a) {
  constexpr int DP = LPC * RPL, P = RPL / 2;     // P: row pairs per lane
  constexpr int kRows = MODE == kMemory ? 2 : 3; // staged rows of DP floats per token
  constexpr int kGroups = 32 / LPC;              // columns groups of a warp
  extern __shared__ float4 smem4[];
  float* smem = reinterpret_cast<float*>(smem4);
  const int stage = stage_floats<MODE, DP>(a.cols);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int l = lane & (LPC - 1);
  const int r = blockIdx.x, h = blockIdx.y, z = blockIdx.z;
  const int kvh = h / (a.N / a.G);
  const Portion po = portion_of(r, a.nd, a.cu_q);
  const int slot = a.slots[r];
  const int c_loc = (warp * kGroups + lane / LPC) * CPT;   // first column of this lane in the block
  const int c0 = z * a.cols + c_loc;
  const int columns = MODE == kMemory ? a.V + 1 : a.V;     // the last one of a memory: normaliser
  if (slot < 0 || slot >= a.num_slots) {                   // padding of a captured batch
    for (int i = 0; i < po.count; ++i)
      for (int c = threadIdx.x; c < a.cols; c += blockDim.x)
        if (z * a.cols + c < a.V)
          a.out[(static_cast<long long>(po.first + i) * a.N + h) * a.V + z * a.cols + c] = 0.0f;
    if (MODE == kMemory && z == 0) {
      for (int i = threadIdx.x; i < po.count; i += blockDim.x) {
        const long long at = static_cast<long long>(po.first + i) * a.N + h;
        a.nq[at] = 0.0f;
        a.low[at] = 1.0f;
      }
    }
    return;
  }
  const bool fresh = a.positions[po.first] == 0;
  const bool warp_on = z * a.cols + warp * kGroups * CPT < columns;    // a column for this warp

  // tokens [i0, i0 + kChunk) of the portion -> stage b: a warp copies the rows of one token at a
  // time (address arithmetic counts here: with few heads a warp has a scheduler for itself)
  const int warps = blockDim.x >> 5;
  const long long qk_step = static_cast<long long>(a.G) * DP, g_step = static_cast<long long>(a.N) * DP;
  const long long v_step = static_cast<long long>(a.N) * a.VP;
  const float* q_src = a.q + po.first * qk_step + kvh * DP + lane * 4;
  const float* k_src = a.k + po.first * qk_step + kvh * DP + lane * 4;
  const float* g_src = MODE != kMemory ? a.g + po.first * g_step + h * DP + lane * 4 : nullptr;
  const float* v_src = a.v + po.first * v_step + static_cast<long long>(h) * a.VP + z * a.cols + lane * 4;
  auto fetch = [&](int i0, int b) {
    const int n = min(kChunk, po.count - i0);
    constexpr int kVec = DP / 4;
    float* dst = smem + b * stage + lane * 4;
#pragma unroll 4
    for (int i = warp; i < n; i += warps) {
      const long long t = i0 + i;
#pragma unroll
      for (int c = 0; c < kVec; c += 32) {
        if (kVec % 32 != 0 && lane + c >= kVec) break;
        copy16(dst + i * DP + c * 4, q_src + t * qk_step + c * 4);
        copy16(dst + (kChunk + i) * DP + c * 4, k_src + t * qk_step + c * 4);
        if (MODE != kMemory) copy16(dst + (2 * kChunk + i) * DP + c * 4, g_src + t * g_step + c * 4);
      }
      float* dv = dst + kRows * kChunk * DP + i * a.cols;
      for (int c = lane * 4; c < a.cols; c += 128) {
        if (z * a.cols + c < a.VP) copy16(dv + c - lane * 4, v_src + t * v_step + c - lane * 4);
        else *reinterpret_cast<float4*>(dv + c - lane * 4) = make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
    float* ss = smem + b * stage + kRows * kChunk * DP + kChunk * a.cols;
    if (threadIdx.x < n) {
      const long long at = static_cast<long long>(po.first + i0 + threadIdx.x) * a.N + h;
      copy4(ss + threadIdx.x, a.s0 + at);
      if (MODE == kMemory) copy4(ss + kChunk + threadIdx.x, a.s1 + at);
    }
  };

  fetch(0, 0);
  copy_commit();

  // state -> registers: lane l holds rows 4 (l + LPC i) .. + 3 of its columns
  float2 S[CPT][P];
  const long long head_at = static_cast<long long>(slot) * a.N + h;
  auto column_state = [&](int c) {
    return MODE == kMemory && c == a.V ? a.vector + head_at * DP
                                       : a.matrix + (head_at * a.V + c) * DP;
  };
#pragma unroll
  for (int j = 0; j < CPT; ++j) {
    const bool in = !fresh && c0 + j < columns;
    const float* src = column_state(c0 + j) + 4 * l;
#pragma unroll
    for (int i = 0; i < P / 2; ++i) {
      Quad u = Quad{both(0.0f), both(0.0f)};
      if (in) u = *reinterpret_cast<const Quad*>(src + 4 * LPC * i);
      S[j][2 * i] = u.x;
      S[j][2 * i + 1] = u.y;
    }
  }
  float m = MODE == kMemory ? a.m0[static_cast<long long>(r) * a.N + h] : 0.0f;

  for (int i0 = 0; i0 < po.count; i0 += kChunk) {
    const int b = (i0 / kChunk) & 1;
    if (i0 + kChunk < po.count) fetch(i0 + kChunk, b ^ 1);
    copy_commit();
    copy_wait<1>();
    __syncthreads();
    const int n = min(kChunk, po.count - i0);
    const float* sq = smem + b * stage + 4 * l;
    const float* sk = sq + kChunk * DP;
    const float* sg = sk + kChunk * DP;                         // not memory
    const float* sv = smem + b * stage + kRows * kChunk * DP;
    const float* ss = sv + kChunk * a.cols;

    // matrix memory: running maximum and the two factors of every token of the chunk, lane t
    // computing token t's
    float keep = 0.0f, add = 0.0f, low = 0.0f;
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
      low = expf(-mt);
      m = __shfl_sync(0xffffffffu, mt, n - 1);
    }

    // gated delta rule: q . k of every token, so that S'^T q = S^T q + (q . k) u needs no second
    // reduction behind the update
    if (MODE == kDelta) {
      float* sqk = smem + b * stage + kRows * kChunk * DP + kChunk * a.cols + kChunk;
      for (int e = threadIdx.x; e < n * 8; e += blockDim.x) {    // eight lanes per token
        const float4* x = reinterpret_cast<const float4*>(smem + b * stage + (e >> 3) * DP);
        const float4* y = x + kChunk * DP / 4;
        float d = 0.0f;
        for (int c = e & 7; c < DP / 4; c += 8) {
          const float4 f = x[c], g = y[c];
          d += f.x * g.x + f.y * g.y + f.z * g.z + f.w * g.w;
        }
        // (n * 8 is a multiple of 8 and so is the block: whole groups take part)
        const unsigned int mask = 0xffu << (lane & 24);
        d += __shfl_xor_sync(mask, d, 1);
        d += __shfl_xor_sync(mask, d, 2);
        d += __shfl_xor_sync(mask, d, 4);
        if ((e & 7) == 0) sqk[e >> 3] = d;
      }
      __syncthreads();
    }

#pragma unroll 2
    for (int i = 0; i < (warp_on ? n : 0); ++i) {
      float v[CPT], o[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) v[j] = sv[i * a.cols + c_loc + j];
      float2 kk[P];
#pragma unroll
      for (int u = 0; u < P / 2; ++u) {
        const Quad x = *reinterpret_cast<const Quad*>(sk + i * DP + 4 * LPC * u);
        kk[2 * u] = x.x; kk[2 * u + 1] = x.y;
      }
      float2 e0[CPT], e1[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) e0[j] = e1[j] = both(0.0f);
      if (MODE == kDelta) {
        const float beta = ss[i], qk = ss[kChunk + i];
        float2 d0[CPT], d1[CPT];
#pragma unroll
        for (int j = 0; j < CPT; ++j) d0[j] = d1[j] = both(0.0f);
#pragma unroll
        for (int u = 0; u < P / 2; ++u) {
          const Quad g = *reinterpret_cast<const Quad*>(sg + i * DP + 4 * LPC * u);
          const Quad q = *reinterpret_cast<const Quad*>(sq + i * DP + 4 * LPC * u);
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            S[j][2 * u] = mul2(S[j][2 * u], g.x);
            S[j][2 * u + 1] = mul2(S[j][2 * u + 1], g.y);
            d0[j] = fma2(S[j][2 * u], kk[2 * u], d0[j]);
            d1[j] = fma2(S[j][2 * u + 1], kk[2 * u + 1], d1[j]);
            e0[j] = fma2(S[j][2 * u], q.x, e0[j]);
            e1[j] = fma2(S[j][2 * u + 1], q.y, e1[j]);
          }
        }
        float d[CPT];
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          d[j] = halves_sum(d0[j]) + halves_sum(d1[j]);
          o[j] = halves_sum(e0[j]) + halves_sum(e1[j]);
        }
#pragma unroll
        for (int w = 1; w < LPC; w <<= 1) {
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            d[j] += __shfl_xor_sync(0xffffffffu, d[j], w);
            o[j] += __shfl_xor_sync(0xffffffffu, o[j], w);
          }
        }
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          const float u1 = beta * (v[j] - d[j]);
          o[j] += qk * u1;
          const float2 u2 = both(u1);
#pragma unroll
          for (int u = 0; u < P; ++u) S[j][u] = fma2(kk[u], u2, S[j][u]);
        }
      } else if (MODE == kWkv) {
        // the read-out is of the state before this token; only it needs the reduction, the state's
        // own chain is one multiply-add per token
#pragma unroll
        for (int u = 0; u < P / 2; ++u) {
          const Quad g = *reinterpret_cast<const Quad*>(sg + i * DP + 4 * LPC * u);
          const Quad q = *reinterpret_cast<const Quad*>(sq + i * DP + 4 * LPC * u);
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            e0[j] = fma2(S[j][2 * u], q.x, e0[j]);
            e1[j] = fma2(S[j][2 * u + 1], q.y, e1[j]);
            const float2 v2 = both(v[j]);
            S[j][2 * u] = fma2(kk[2 * u], v2, mul2(S[j][2 * u], g.x));
            S[j][2 * u + 1] = fma2(kk[2 * u + 1], v2, mul2(S[j][2 * u + 1], g.y));
          }
        }
#pragma unroll
        for (int j = 0; j < CPT; ++j) o[j] = halves_sum(e0[j]) + halves_sum(e1[j]);
#pragma unroll
        for (int w = 1; w < LPC; w <<= 1) {
#pragma unroll
          for (int j = 0; j < CPT; ++j) o[j] += __shfl_xor_sync(0xffffffffu, o[j], w);
        }
        const float now = ss[i];
#pragma unroll
        for (int j = 0; j < CPT; ++j) o[j] += now * v[j];
      } else {
        const float2 a2 = both(__shfl_sync(0xffffffffu, keep, i));
        const float b1 = __shfl_sync(0xffffffffu, add, i);
        float2 v2[CPT];
#pragma unroll
        for (int j = 0; j < CPT; ++j) v2[j] = both(b1 * v[j]);
#pragma unroll
        for (int u = 0; u < P / 2; ++u) {
          const Quad q = *reinterpret_cast<const Quad*>(sq + i * DP + 4 * LPC * u);
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            S[j][2 * u] = fma2(kk[2 * u], v2[j], mul2(S[j][2 * u], a2));
            S[j][2 * u + 1] = fma2(kk[2 * u + 1], v2[j], mul2(S[j][2 * u + 1], a2));
            e0[j] = fma2(S[j][2 * u], q.x, e0[j]);
            e1[j] = fma2(S[j][2 * u + 1], q.y, e1[j]);
          }
        }
#pragma unroll
        for (int j = 0; j < CPT; ++j) o[j] = halves_sum(e0[j]) + halves_sum(e1[j]);
#pragma unroll
        for (int w = 1; w < LPC; w <<= 1) {
#pragma unroll
          for (int j = 0; j < CPT; ++j) o[j] += __shfl_xor_sync(0xffffffffu, o[j], w);
        }
      }
      const long long at = static_cast<long long>(po.first + i0 + i) * a.N + h;
      if (l == 0) {
#pragma unroll
        for (int j = 0; j < CPT; ++j) {
          if (c0 + j < a.V) a.out[at * a.V + c0 + j] = o[j];
          else if (MODE == kMemory && c0 + j == a.V) a.nq[at] = o[j];
        }
      }
    }
    if (MODE == kMemory && z == 0 && warp == 0 && lane < n)
      a.low[static_cast<long long>(po.first + i0 + lane) * a.N + h] = low;
    __syncthreads();           // stage b is refilled next
  }

  // registers -> state
#pragma unroll
  for (int j = 0; j < CPT; ++j) {
    if (c0 + j >= columns) continue;
    float* dst = column_state(c0 + j) + 4 * l;
#pragma unroll
    for (int i = 0; i < P / 2; ++i)
      *reinterpret_cast<Quad*>(dst + 4 * LPC * i) =
          Quad{S[j][2 * i], S[j][2 * i + 1]};
  }
  if (MODE == kMemory) {
    if (z == 0 && threadIdx.x == 0) a.scalar[head_at] = m;
  } else if (MODE == kDelta && z == 0 && a.ntaps > 1) {
    if (a.elt == 2) keep_taps<uint16_t>(a, po, slot, h);
    else keep_taps<uint32_t>(a, po, slot, h);
  }
}

template <int MODE, int LPC, int RPL, int CPT>
static int launch_scan(ScanArgs& a, int requests, int warps, cudaStream_t s) {
  constexpr int kPerWarp = 32 / LPC * CPT;
  const int columns = MODE == kMemory ? a.V + 1 : a.V;
  const int want = (columns + kPerWarp - 1) / kPerWarp;
  if (warps > want) warps = want;
  a.cols = warps * kPerWarp;
  const int smem = 2 * stage_floats<MODE, LPC * RPL>(a.cols) * static_cast<int>(sizeof(float));
  static bool done[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return -9;
  if (!done[dev]) {
    cudaError_t e = cudaFuncSetAttribute(recurrent_scan_kernel<MODE, LPC, RPL, CPT>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    done[dev] = true;
  }
  dim3 grid(requests, a.N, (columns + a.cols - 1) / a.cols);
  recurrent_scan_kernel<MODE, LPC, RPL, CPT><<<grid, warps * 32, smem, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

// A warp of the wide form walks 32 (DP <= 128) or 16 columns, one of the narrow forms 8 or 4: the
// widest form that gives every scheduler of the GPU a warp.
template <int MODE, int DP>
static int dispatch_scan(ScanArgs& a, int requests, cudaStream_t s) {
  constexpr int kWide = DP <= 128 ? 2 : 4;
  const long long heads = static_cast<long long>(requests) * a.N;
  const long long schedulers = 4ll * sm_count();
  const auto warps = [&](int per) { return heads * ((a.V + per - 1) / per); };
  if (warps(64 / kWide) >= schedulers)
    return launch_scan<MODE, kWide, DP / kWide, 2>(a, requests, 4, s);
  if (warps(8) >= schedulers) return launch_scan<MODE, 8, DP / 8, 2>(a, requests, 4, s);
  return launch_scan<MODE, 8, DP / 8, 1>(a, requests, 4, s);
}

template <int MODE>
static int dispatch_scan(ScanArgs& a, int DP, int requests, cudaStream_t s) {
  switch (DP) {
    case 32: return dispatch_scan<MODE, 32>(a, requests, s);
    case 64: return dispatch_scan<MODE, 64>(a, requests, s);
    case 96: return dispatch_scan<MODE, 96>(a, requests, s);
    case 128: return dispatch_scan<MODE, 128>(a, requests, s);
    case 192: return dispatch_scan<MODE, 192>(a, requests, s);
    case 256: return dispatch_scan<MODE, 256>(a, requests, s);
  }
  return -20;
}

// ---------------------------------------------------------------------------
struct HeadNormArgs {
  const float* o;            // [T, N, V]
  const float *nq, *low;     // [T, N]: o is divided by max(|nq|, low) + 1e-6 first, or null
  const float* w;            // norm weight: [V] shared by the heads, or [N * V]
  const void* z;             // [T, N * V] gate projection, row pitch ldz
  void* out;                 // [T, N * V], row pitch ldo
  long long ldz, ldo;
  int T, N, V, per_head, silu;
  float eps, scale;
};

template <typename T, int W>
__device__ __forceinline__ void store_t(T* p, const float (&f)[W]) {
  if constexpr (W == 4 && sizeof(T) == 2) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  } else if constexpr (W == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    p[0] = from_f32<T>(f[0]);
  }
}

// One warp per row and head.
template <typename T, int W>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const HeadNormArgs a) {
  const int lane = threadIdx.x & 31;
  const long long row = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (row >= static_cast<long long>(a.T) * a.N) return;
  const long long t = row / a.N;
  const int h = static_cast<int>(row - t * a.N);
  const float* o = a.o + row * a.V;
  const float* w = a.w + (a.per_head ? h * a.V : 0);
  const T* z = static_cast<const T*>(a.z) + t * a.ldz + h * a.V;
  T* out = static_cast<T*>(a.out) + t * a.ldo + h * a.V;
  constexpr int kKeep = W == 4 ? 2 : 8;          // vectors per lane that stay in registers
  float f[kKeep][W], g[kKeep][W], ss = 0.0f;
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = (lane + 32 * i) * W;
    if (c >= a.V) continue;
    load_n<float, W>(o + c, f[i]);
    load_n<T, W>(z + c, g[i]);
  }
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    if ((lane + 32 * i) * W >= a.V) continue;
#pragma unroll
    for (int j = 0; j < W; ++j) ss += f[i][j] * f[i][j];
  }
  for (int c = (lane + 32 * kKeep) * W; c < a.V; c += 32 * W) {
    float x[W];
    load_n<float, W>(o + c, x);
#pragma unroll
    for (int j = 0; j < W; ++j) ss += x[j] * x[j];
  }
  const float den = a.nq != nullptr ? 1.0f / (fmaxf(fabsf(a.nq[row]), a.low[row]) + 1e-6f) : 1.0f;
  const float inv =
      den * (1.0f / sqrtf(warp_sum(ss) * den * den / static_cast<float>(a.V) + a.eps)) * a.scale;
  auto put = [&](int c, float (&x)[W], const float (&gate)[W]) {
    float b[W];
    load_n<float, W>(w + c, b);
#pragma unroll
    for (int j = 0; j < W; ++j) x[j] = x[j] * inv * b[j] * (a.silu ? silu<T>(gate[j]) : sigmoid_t<T>(gate[j]));
    store_t<T, W>(out + c, x);
  };
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = (lane + 32 * i) * W;
    if (c < a.V) put(c, f[i], g[i]);
  }
  for (int c = (lane + 32 * kKeep) * W; c < a.V; c += 32 * W) {
    float x[W], gate[W];
    load_n<float, W>(o + c, x);
    load_n<T, W>(z + c, gate);
    put(c, x, gate);
  }
}

// ---------------------------------------------------------------------------
// Requests that bring one token: everything between the wide projections and the output projection
// in one CTA per (request, head), 256 threads.
struct StepArgs {
  const void* hrow;          // [nd, H] mixer input, row pitch ldh
  const void* x[3];          // q, k, v projections, row pitch ld
  const void* gate;          // [nd, N V] output gate projection, row pitch ldg
  const float* z;            // delta: decay projection [nd, N D], row pitch ldz
                             // wkv: inner row of the decay's projection [nd, H]
  const void *w0, *w1;       // rows [N, H]: delta step size, - ; memory input gate, forget gate
                             // wkv: second step of the decay's projection [N D, H], -
  const float *b0, *b1;      // memory: their biases [N]; wkv: decay base, bonus [N D]
  const float* taps_w[3];    // delta: convolution weights
  const float *dt_bias, *a_log;
  const float* norm;         // [V], or [N V] with per_head
  void* taps;
  float *matrix, *vector, *scalar;
  void* out;                 // [nd, N V], row pitch ldo
  const long long* positions;
  const int* slots;
  long long ldh, ld, ldz, ldg, ldo;
  int H, G, N, D, V, ntaps, num_slots, per_head;
  float cap, qscale, eps, scale;
};

// 8 elements as floats (16-byte aligned)
template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&f)[8]) {
  if constexpr (sizeof(T) == 2) {
    vec8_load<T>(p, f);
  } else {
    const float4 a = *reinterpret_cast<const float4*>(p);
    const float4 b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
}

// This thread's share of x . w over n elements (vec: both 16-byte aligned and n a multiple of 8).
template <typename T>
__device__ __forceinline__ float dot_share(const T* x, const T* w, int n, bool vec) {
  float s = 0.0f;
  if (vec) {
    for (int c = threadIdx.x * 8; c < n; c += blockDim.x * 8) {
      float f[8], g[8];
      load8<T>(x + c, f);
      load8<T>(w + c, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) s += f[i] * g[i];
    }
  } else {
    for (int c = threadIdx.x; c < n; c += blockDim.x) s += to_f32<T>(x[c]) * to_f32<T>(w[c]);
  }
  return s;
}

// inner: wkv's decay rank
__host__ __device__ inline int step_floats(int DP, int V, int inner) {
  return 3 * DP + 3 * ((V + 3) / 4 * 4) + 64 + inner;
}

template <typename T, int MODE, int RPL, int CPT>
__global__ void __launch_bounds__(256, RPL < 32 ? 2 : 1) recurrent_step_kernel(const StepArgs a) {
  constexpr int DP = 8 * RPL, P = RPL / 2;
  constexpr int kCols = 8 * 4 * CPT;              // columns per pass
  extern __shared__ float4 smem4[];
  float* sq = reinterpret_cast<float*>(smem4);    // [DP]
  float* sk = sq + DP;                            // [DP]
  float* sg = sk + DP;                            // [DP] decays (delta), normaliser products (memory)
  const int VS = (a.V + 3) / 4 * 4;
  float* sv = sg + DP;                            // [V]
  float* so = sv + VS;                            // [V]
  float* sz = so + VS;                            // [V] output gate
  float* red = sz + VS;                           // [64]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l = lane & 7;
  const int r = blockIdx.x, h = blockIdx.y;
  const int kvh = h / (a.N / a.G);
  T* out = static_cast<T*>(a.out) + static_cast<long long>(r) * a.ldo + h * a.V;
  const int slot = a.slots[r];
  if (slot < 0 || slot >= a.num_slots) {          // padding of a captured batch
    for (int c = tid; c < a.V; c += blockDim.x) out[c] = from_f32<T>(0.0f);
    return;
  }
  const long long pos = a.positions[r];
  const bool fresh = pos == 0;
  const long long head_at = static_cast<long long>(slot) * a.N + h;
  const int c_warp = (warp * 4 + (lane >> 3)) * CPT;

  float2 S[CPT][P];
  auto load_state = [&](int base) {
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
      const int c = base + c_warp + j;
      const bool in = !fresh && c < a.V;
      const float* src = a.matrix + (head_at * a.V + c) * DP + 4 * l;
#pragma unroll
      for (int i = 0; i < P / 2; ++i) {
        Quad u = Quad{both(0.0f), both(0.0f)};
        if (in) u = *reinterpret_cast<const Quad*>(src + 32 * i);
        S[j][2 * i] = u.x;
        S[j][2 * i + 1] = u.y;
      }
    }
  };
  load_state(0);                                  // in flight while the inputs are computed

  const T* hr = MODE == kWkv ? nullptr
                             : static_cast<const T*>(a.hrow) + static_cast<long long>(r) * a.ldh;
  const bool vec = (a.H % 8) == 0 && ((reinterpret_cast<uintptr_t>(hr) |
                                       reinterpret_cast<uintptr_t>(a.w0) |
                                       reinterpret_cast<uintptr_t>(a.w1)) & 15) == 0;
  const long long xrow = static_cast<long long>(r) * a.ld;
  float d0 = 0.0f;
  if (MODE != kWkv)
    d0 = dot_share<T>(hr, static_cast<const T*>(a.w0) + static_cast<long long>(h) * a.H, a.H, vec);
  float d1 = 0.0f;
  if (MODE == kMemory)
    d1 = dot_share<T>(hr, static_cast<const T*>(a.w1) + static_cast<long long>(h) * a.H, a.H, vec);

  const T* gz = static_cast<const T*>(a.gate) + static_cast<long long>(r) * a.ldg + h * a.V;
  for (int c = tid; c < a.V; c += blockDim.x) {
    const float g = to_f32<T>(gz[c]);
    sz[c] = MODE == kWkv ? silu<T>(g) : sigmoid_t<T>(g);
  }
  if (MODE == kDelta) {
    const int C = 2 * a.G * a.D + a.N * a.V;
    const T* ring = static_cast<const T*>(a.taps) + static_cast<long long>(slot) * a.ntaps * C;
    const float rate = expf(a.a_log[h]);
    const float* z = a.z + r * a.ldz + h * a.D;
    for (int d = tid; d < DP; d += blockDim.x)
      sg[d] = d < a.D ? exp_t<T>(-rate * softplus_t<T>(z[d] + a.dt_bias[h * a.D + d])) : 0.0f;
    for (int e = tid; e < 2 * DP + a.V; e += blockDim.x) {
      const int which = e < DP ? 0 : e < 2 * DP ? 1 : 2;
      const int d = which == 0 ? e : which == 1 ? e - DP : e - 2 * DP;
      const int head = which == 2 ? h : kvh, dim = which == 2 ? a.V : a.D;
      float f = 0.0f;
      if (d < dim) {
        const int ch = head * dim + d;
        const int at = ch + (which == 0 ? 0 : which == 1 ? a.G * a.D : 2 * a.G * a.D);
        const float* w = a.taps_w[which] + ch;
        const int wld = (which == 2 ? a.N : a.G) * dim;
        float s = w[(a.ntaps - 1) * wld] * to_f32<T>(static_cast<const T*>(a.x[which])[xrow + ch]);
#pragma unroll 3
        for (int o = 1; o < a.ntaps; ++o)
          if (pos - o >= 0)
            s += w[(a.ntaps - 1 - o) * wld] * to_f32<T>(ring[(pos - o) % a.ntaps * C + at]);
        f = silu<T>(s);
      }
      (which == 0 ? sq : which == 1 ? sk : sv)[d] = f;
    }
  } else {
    for (int d = tid; d < DP; d += blockDim.x) {
      const bool in = d < a.D;
      sq[d] = in ? to_f32<T>(static_cast<const T*>(a.x[0])[xrow + h * a.D + d]) * a.qscale : 0.0f;
      sk[d] = in ? to_f32<T>(static_cast<const T*>(a.x[1])[xrow + h * a.D + d]) : 0.0f;
    }
    for (int c = tid; c < a.V; c += blockDim.x)
      sv[c] = to_f32<T>(static_cast<const T*>(a.x[2])[xrow + h * a.V + c]);
  }
  if (MODE == kWkv) {                             // inner row of the decay's projection
    float* st = red + 64;
    for (int c = tid; c < a.H; c += blockDim.x) st[c] = tanhf(a.z[r * a.ldz + c]);
  }
  const float z0 = block_sum(d0, red);            // (synchronises: the shared rows are complete)
  const float z1 = MODE == kMemory ? block_sum(d1, red) : 0.0f;

  float beta = 0.0f, keep = 0.0f, add = 0.0f, den = 1.0f, now = 0.0f;
  if (MODE == kDelta) {
    beta = sigmoid(z0);
    if (warp < 2) {                               // unit vectors
      float* x = warp == 0 ? sq : sk;
      float ss = 0.0f;
      for (int d = lane; d < DP; d += 32) ss += x[d] * x[d];
      float inv = 1.0f / sqrtf(warp_sum(ss) + 1e-6f);
      if (warp == 0) inv *= 1.0f / sqrtf(static_cast<float>(a.D));
      for (int d = lane; d < DP; d += 32) x[d] *= inv;
    } else if (a.ntaps > 1) {                     // this token's row of the convolution state
      const int C = 2 * a.G * a.D + a.N * a.V;
      T* row = static_cast<T*>(a.taps) + (static_cast<long long>(slot) * a.ntaps + pos % a.ntaps) * C;
      for (int d = tid - 64; d < a.V; d += blockDim.x - 64)
        row[2 * a.G * a.D + h * a.V + d] = static_cast<const T*>(a.x[2])[xrow + h * a.V + d];
      if (h % (a.N / a.G) == 0) {
        for (int d = tid - 64; d < a.D; d += blockDim.x - 64) {
          row[kvh * a.D + d] = static_cast<const T*>(a.x[0])[xrow + kvh * a.D + d];
          row[(a.G + kvh) * a.D + d] = static_cast<const T*>(a.x[1])[xrow + kvh * a.D + d];
        }
      }
    }
    __syncthreads();
  } else if (MODE == kWkv) {
    const float* st = red + 64;
    float part = 0.0f;
    for (int d = tid; d < a.D; d += blockDim.x) part += sq[d] * sk[d] * a.b1[h * a.D + d];
    // decays: four threads a channel, 8 inner columns at a time
    for (int base = 0; base < DP; base += 64) {
      const int d = base + (tid >> 2);
      float s = 0.0f;
      if (d < a.D) {
        const T* w = static_cast<const T*>(a.w0) + (static_cast<long long>(h) * a.D + d) * a.H;
        for (int c = (tid & 3) * 8; c < a.H; c += 32) {
          float f[8];
          load8<T>(w + c, f);
#pragma unroll
          for (int i = 0; i < 8; ++i) s += f[i] * st[c + i];
        }
      }
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s += __shfl_xor_sync(0xffffffffu, s, 2);
      if ((tid & 3) == 0 && d < DP)
        sg[d] = d < a.D ? exp_t<T>(-exp_t<T>(s + a.b0[h * a.D + d])) : 0.0f;
    }
    now = block_sum(part, red);                   // (synchronises: the decays are complete)
  } else {
    const float li = soft_cap(z0 + a.b0[h], a.cap);
    const float lf = -softplus(-soft_cap(z1 + a.b1[h], a.cap));
    const float m = fresh ? 0.0f : a.scalar[head_at];
    const float mt = fmaxf(lf + m, li);
    keep = expf(lf + (m - mt));
    add = expf(li - mt);
    float part = 0.0f;
    for (int d = tid; d < DP; d += blockDim.x) {
      float* n = a.vector + head_at * DP + d;
      const float v = (fresh ? 0.0f : keep * *n) + add * sk[d];
      *n = v;
      part += v * sq[d];
    }
    den = 1.0f / (fmaxf(fabsf(block_sum(part, red)), expf(-mt)) + 1e-6f);
    if (tid == 0) a.scalar[head_at] = mt;         // every thread has read m (block_sum)
  }

  float ss = 0.0f;
  for (int base = 0; base < a.V; base += kCols) {
    if (base > 0) load_state(base);
    const int c0 = base + c_warp;
    float v[CPT], o[CPT], d[CPT];
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
      v[j] = c0 + j < a.V ? sv[c0 + j] : 0.0f;
      float2 e0 = both(0.0f), e1 = both(0.0f);
      if (MODE == kDelta) {
#pragma unroll
        for (int u = 0; u < P / 2; ++u) {
          const Quad g = *reinterpret_cast<const Quad*>(sg + 4 * l + 32 * u);
          const Quad k = *reinterpret_cast<const Quad*>(sk + 4 * l + 32 * u);
          S[j][2 * u] = mul2(S[j][2 * u], g.x);
          S[j][2 * u + 1] = mul2(S[j][2 * u + 1], g.y);
          e0 = fma2(S[j][2 * u], k.x, e0);
          e1 = fma2(S[j][2 * u + 1], k.y, e1);
        }
      }
      d[j] = halves_sum(e0) + halves_sum(e1);
    }
    if (MODE == kDelta) {
#pragma unroll
      for (int w = 1; w < 8; w <<= 1) {
#pragma unroll
        for (int j = 0; j < CPT; ++j) d[j] += __shfl_xor_sync(0xffffffffu, d[j], w);
      }
    }
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
      const float2 u2 = both(MODE == kDelta ? beta * (v[j] - d[j]) : MODE == kWkv ? v[j] : add * v[j]);
      const float2 a2 = both(keep);
      float2 e0 = both(0.0f), e1 = both(0.0f);
#pragma unroll
      for (int u = 0; u < P / 2; ++u) {
        if (MODE == kWkv) {                       // the read-out is of the state before this token
          const Quad g = *reinterpret_cast<const Quad*>(sg + 4 * l + 32 * u);
          const Quad k = *reinterpret_cast<const Quad*>(sk + 4 * l + 32 * u);
          const Quad q = *reinterpret_cast<const Quad*>(sq + 4 * l + 32 * u);
          e0 = fma2(S[j][2 * u], q.x, e0);
          e1 = fma2(S[j][2 * u + 1], q.y, e1);
          S[j][2 * u] = fma2(k.x, u2, mul2(S[j][2 * u], g.x));
          S[j][2 * u + 1] = fma2(k.y, u2, mul2(S[j][2 * u + 1], g.y));
          continue;
        }
        const Quad k = *reinterpret_cast<const Quad*>(sk + 4 * l + 32 * u);
        const Quad q = *reinterpret_cast<const Quad*>(sq + 4 * l + 32 * u);
        if (MODE == kMemory) {
          S[j][2 * u] = mul2(S[j][2 * u], a2);
          S[j][2 * u + 1] = mul2(S[j][2 * u + 1], a2);
        }
        S[j][2 * u] = fma2(k.x, u2, S[j][2 * u]);
        S[j][2 * u + 1] = fma2(k.y, u2, S[j][2 * u + 1]);
        e0 = fma2(S[j][2 * u], q.x, e0);
        e1 = fma2(S[j][2 * u + 1], q.y, e1);
      }
      o[j] = halves_sum(e0) + halves_sum(e1);
      if (c0 + j < a.V) {
        float* dst = a.matrix + (head_at * a.V + c0 + j) * DP + 4 * l;
#pragma unroll
        for (int i = 0; i < P / 2; ++i)
          *reinterpret_cast<Quad*>(dst + 32 * i) =
              Quad{S[j][2 * i], S[j][2 * i + 1]};
      }
    }
#pragma unroll
    for (int w = 1; w < 8; w <<= 1) {
#pragma unroll
      for (int j = 0; j < CPT; ++j) o[j] += __shfl_xor_sync(0xffffffffu, o[j], w);
    }
    if (l == 0) {
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
        if (c0 + j >= a.V) continue;
        o[j] = o[j] * den + now * v[j];
        so[c0 + j] = o[j];
        ss += o[j] * o[j];
      }
    }
  }
  ss = block_sum(ss, red);                        // (synchronises: so is complete)
  const float inv = 1.0f / sqrtf(ss / static_cast<float>(a.V) + a.eps) * a.scale;
  const float* nw = a.norm + (a.per_head ? h * a.V : 0);
  for (int c = tid; c < a.V; c += blockDim.x)
    out[c] = from_f32<T>(so[c] * inv * nw[c] * sz[c]);
}

template <typename T, int MODE, int RPL, int CPT>
static int launch_step(const StepArgs& a, int requests, cudaStream_t s) {
  const int smem = step_floats(8 * RPL, a.V, MODE == kWkv ? a.H : 0) * static_cast<int>(sizeof(float));
  if (smem > 48 * 1024) return -20;
  recurrent_step_kernel<T, MODE, RPL, CPT><<<dim3(requests, a.N), 256, smem, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int MODE>
static int dispatch_step(const StepArgs& a, int DP, int requests, cudaStream_t s) {
  switch (DP) {
    case 32: return launch_step<T, MODE, 4, 4>(a, requests, s);
    case 64: return launch_step<T, MODE, 8, 4>(a, requests, s);
    case 96: return launch_step<T, MODE, 12, 4>(a, requests, s);
    case 128: return launch_step<T, MODE, 16, 4>(a, requests, s);
    case 192: return launch_step<T, MODE, 24, 2>(a, requests, s);
    case 256: return launch_step<T, MODE, 32, 2>(a, requests, s);
  }
  return -20;
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
  // few tokens: the items of a strip go to several CTAs
  const int strips = (T + kStrip - 1) / kStrip, most = (2 * G + 2 * N + 7) / 8;
  int split = (4 * sm_count() + strips - 1) / strips;
  if (split > most) split = most;
  const dim3 grid(strips, split);
  const uintptr_t x = reinterpret_cast<uintptr_t>(xq) | reinterpret_cast<uintptr_t>(xk) |
                      reinterpret_cast<uintptr_t>(xv) | reinterpret_cast<uintptr_t>(taps);
  const bool v4 = (D % 4) == 0 && (V % 4) == 0 && (VP % 4) == 0 && (ld % 4) == 0 &&
                  (ldz % 4) == 0 && (x % (dtype == 0 ? 8 : 16)) == 0 &&
                  ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(wq) |
                    reinterpret_cast<uintptr_t>(wk) | reinterpret_cast<uintptr_t>(wv)) % 16) == 0;
#define B200_IN(NT, W)                                                             \
  do {                                                                             \
    if (dtype == 0) delta_inputs_kernel<__nv_bfloat16, NT, W><<<grid, 256, 0, s>>>(a); \
    else delta_inputs_kernel<float, NT, W><<<grid, 256, 0, s>>>(a);                 \
  } while (0)
  if (ntaps <= 4) {
    if (v4) B200_IN(4, 4);
    else B200_IN(4, 1);
  } else {
    if (v4) B200_IN(8, 4);
    else B200_IN(8, 1);
  }
#undef B200_IN
  return static_cast<int>(cudaGetLastError());
}

// fp32 inputs and log gates of the matrix memory; VP > V (column V of vo is the normaliser's 1).
// dtype (of q, k, v): 0 bf16, 2 fp32.
B200_API int b200_memory_inputs(const void* q, const void* k, const void* v, long long ld,
                                const float* zi, const float* zf, long long ldg, const float* ib,
                                const float* fb, const float* scalar, float cap, float qscale,
                                float* qo, float* ko, float* vo, float* io, float* fo, float* m0,
                                const long long* positions, const int* slots, int num_slots,
                                const int* cu_q, int T, int N, int D, int V, int DP, int VP,
                                int nd, int np, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (N <= 0 || D <= 0 || D > DP || V <= 0 || V >= VP || (dtype != 0 && dtype != 2)) return -2;
  MemoryIn a;
  a.q = q; a.k = k; a.v = v; a.zi = zi; a.zf = zf; a.ib = ib; a.fb = fb; a.scalar = scalar;
  a.qo = qo; a.ko = ko; a.vo = vo; a.io = io; a.fo = fo; a.m0 = m0; a.positions = positions;
  a.slots = slots; a.cu_q = cu_q; a.ld = ld; a.ldg = ldg; a.T = T; a.N = N; a.D = D; a.V = V;
  a.DP = DP; a.VP = VP; a.num_slots = num_slots; a.nd = nd; a.np = np; a.cap = cap;
  a.qscale = qscale;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const uintptr_t x = reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) |
                      reinterpret_cast<uintptr_t>(v);
  const bool v4 = (D % 4) == 0 && (V % 4) == 0 && (VP % 4) == 0 && (ld % 4) == 0 &&
                  (x % (dtype == 0 ? 8 : 16)) == 0;
  if (dtype == 0) {
    if (v4) memory_inputs_kernel<__nv_bfloat16, 4><<<T, 256, 0, s>>>(a);
    else memory_inputs_kernel<__nv_bfloat16, 1><<<T, 256, 0, s>>>(a);
  } else {
    if (v4) memory_inputs_kernel<float, 4><<<T, 256, 0, s>>>(a);
    else memory_inputs_kernel<float, 1><<<T, 256, 0, s>>>(a);
  }
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

// Matrix memory over the portions of a step; the state is (matrix, vector n, scalar m).  `out` is
// the undivided read-out, nq and low what b200_head_norm_gate divides it by.
B200_API int b200_memory_scan(const float* q, const float* k, const float* v, const float* li,
                              const float* lf, const float* m0, float* out, float* nq, float* low,
                              float* matrix, float* vector, float* scalar,
                              const long long* positions, const int* slots, int num_slots,
                              const int* cu_q, int N, int D, int V, int DP, int VP, int nd, int np,
                              void* stream) {
  if (nd + np <= 0) return 0;
  if (N <= 0 || (VP % 4) != 0 || VP <= V) return -2;
  ScanArgs a{};
  a.q = q; a.k = k; a.v = v; a.s0 = li; a.s1 = lf; a.m0 = m0; a.out = out; a.nq = nq; a.low = low;
  a.matrix = matrix; a.vector = vector; a.scalar = scalar; a.positions = positions;
  a.slots = slots; a.num_slots = num_slots; a.cu_q = cu_q; a.G = N; a.N = N; a.D = D; a.V = V;
  a.VP = VP; a.nd = nd; a.np = np; a.ntaps = 1;
  return dispatch_scan<kMemory>(a, DP, nd + np, static_cast<cudaStream_t>(stream));
}

// out = o' / rms(o') per head * w * sigmoid(z) (silu 1: SiLU(z)) * scale with o' = o, or with nq and
// low o / (max(|nq|, low) + 1e-6).  per_head: w is [N * V], else [V].  dtype (of z and out): 0 bf16,
// 2 fp32.
B200_API int b200_head_norm_gate(const float* o, const float* nq, const float* low, const float* w,
                                 int per_head, const void* z, long long ldz, void* out,
                                 long long ldo, float eps, float scale, int T, int N, int V,
                                 int silu, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (N <= 0 || V <= 0 || (dtype != 0 && dtype != 2)) return -2;
  HeadNormArgs a;
  a.silu = silu;
  a.o = o; a.nq = nq; a.low = low; a.w = w; a.z = z; a.out = out; a.ldz = ldz; a.ldo = ldo;
  a.T = T; a.N = N; a.V = V; a.per_head = per_head; a.eps = eps; a.scale = scale;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int blocks = static_cast<int>((static_cast<long long>(T) * N + 7) / 8);
  const uintptr_t lo = reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out);
  const uintptr_t hi = reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(w);
  const bool v4 = (V % 4) == 0 && (ldz % 4) == 0 && (ldo % 4) == 0 && (hi % 16) == 0 &&
                  (lo % (dtype == 0 ? 8 : 16)) == 0;
  if (dtype == 0) {
    if (v4) head_norm_gate_kernel<__nv_bfloat16, 4><<<blocks, 256, 0, s>>>(a);
    else head_norm_gate_kernel<__nv_bfloat16, 1><<<blocks, 256, 0, s>>>(a);
  } else {
    if (v4) head_norm_gate_kernel<float, 4><<<blocks, 256, 0, s>>>(a);
    else head_norm_gate_kernel<float, 1><<<blocks, 256, 0, s>>>(a);
  }
  return static_cast<int>(cudaGetLastError());
}

// One token of `nd` requests through the gated delta rule, from the projections to the gated
// output: z [nd, N D] fp32 is the decay's projection, gate [nd, N V] the output gate's, wb [N, H] the
// weights of the step size's.  dtype: 0 bf16, 2 fp32.  -20: not covered (very wide heads).
B200_API int b200_delta_step(const void* h, long long ldh, int H, const void* xq, const void* xk,
                             const void* xv, long long ld, const float* z, long long ldz,
                             const void* gate, long long ldg, const void* wb, const float* wq,
                             const float* wk, const float* wv, int ntaps, const float* dt_bias,
                             const float* a_log, const float* norm, void* taps, float* matrix,
                             const long long* positions, const int* slots, int num_slots, void* out,
                             long long ldo, float eps, float scale, int nd, int G, int N, int D,
                             int V, int DP, int dtype, void* stream) {
  if (nd <= 0) return 0;
  if (G <= 0 || N <= 0 || N % G != 0 || D <= 0 || D > DP || V <= 0 || H <= 0 || ntaps < 1 ||
      (dtype != 0 && dtype != 2))
    return -2;
  StepArgs a{};
  a.hrow = h; a.ldh = ldh; a.H = H; a.x[0] = xq; a.x[1] = xk; a.x[2] = xv; a.ld = ld; a.z = z;
  a.ldz = ldz; a.gate = gate; a.ldg = ldg; a.w0 = wb; a.taps_w[0] = wq; a.taps_w[1] = wk;
  a.taps_w[2] = wv; a.ntaps = ntaps; a.dt_bias = dt_bias; a.a_log = a_log; a.norm = norm;
  a.taps = taps; a.matrix = matrix; a.positions = positions; a.slots = slots;
  a.num_slots = num_slots; a.out = out; a.ldo = ldo; a.eps = eps; a.scale = scale; a.G = G;
  a.N = N; a.D = D; a.V = V;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == 0 ? dispatch_step<__nv_bfloat16, kDelta>(a, DP, nd, s)
                    : dispatch_step<float, kDelta>(a, DP, nd, s);
}

// The same for the matrix memory: wi, wf [N, H] are the gates' projections, `gate` (a view of the
// same rows as q, k, v) the output gate's result.
B200_API int b200_memory_step(const void* h, long long ldh, int H, const void* xq, const void* xk,
                              const void* xv, const void* gate, long long ld, const void* wi,
                              const void* wf, const float* ib, const float* fb, float cap,
                              float qscale, const float* norm, float* matrix, float* vector,
                              float* scalar, const long long* positions, const int* slots,
                              int num_slots, void* out, long long ldo, float eps, float scale,
                              int nd, int N, int D, int V, int DP, int dtype, void* stream) {
  if (nd <= 0) return 0;
  if (N <= 0 || D <= 0 || D > DP || V <= 0 || H <= 0 || (dtype != 0 && dtype != 2)) return -2;
  StepArgs a{};
  a.hrow = h; a.ldh = ldh; a.H = H; a.x[0] = xq; a.x[1] = xk; a.x[2] = xv; a.gate = gate;
  a.ldg = ld; a.ld = ld; a.w0 = wi; a.w1 = wf; a.b0 = ib; a.b1 = fb; a.cap = cap; a.qscale = qscale;
  a.norm = norm; a.per_head = 1; a.matrix = matrix; a.vector = vector; a.scalar = scalar;
  a.positions = positions; a.slots = slots; a.num_slots = num_slots; a.out = out; a.ldo = ldo;
  a.eps = eps; a.scale = scale; a.G = N; a.N = N; a.D = D; a.V = V;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == 0 ? dispatch_step<__nv_bfloat16, kMemory>(a, DP, nd, s)
                    : dispatch_step<float, kMemory>(a, DP, nd, s);
}

// fp32 inputs of time mixing: ro, ko, go [T, N, DP], vo [T, N, VP], now [T, N]; z [T, N * D] is the
// decay's projection, decays are exp(-exp(z + base)).  dtype (of r, k, v): 0 bf16, 2 fp32.
B200_API int b200_wkv_inputs(const void* r, const void* k, const void* v, long long ld,
                             const float* z, long long ldz, const float* base, const float* bonus,
                             float* ro, float* ko, float* go, float* vo, float* now, int T, int N,
                             int D, int DP, int VP, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (N <= 0 || D <= 0 || D > DP || DP > 256 || VP < D || VP > DP || (VP % 4) != 0 ||
      (dtype != 0 && dtype != 2))
    return -2;
  WkvIn a;
  a.r = r; a.k = k; a.v = v; a.z = z; a.base = base; a.bonus = bonus; a.ro = ro; a.ko = ko;
  a.go = go; a.vo = vo; a.now = now; a.ld = ld; a.ldz = ldz; a.T = T; a.N = N; a.D = D; a.DP = DP;
  a.VP = VP;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const uintptr_t x = reinterpret_cast<uintptr_t>(r) | reinterpret_cast<uintptr_t>(k) |
                      reinterpret_cast<uintptr_t>(v);
  const uintptr_t f = reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(base) |
                      reinterpret_cast<uintptr_t>(bonus);
  const bool v4 = (D % 4) == 0 && (ld % 4) == 0 && (ldz % 4) == 0 &&
                  (x % (dtype == 0 ? 8 : 16)) == 0 && (f % 16) == 0;
  const auto blocks = [&](int lanes) {
    return static_cast<unsigned int>((static_cast<long long>(T) * N * lanes + 255) / 256);
  };
#define B200_WI(TT)                                                            \
  do {                                                                         \
    if (!v4) wkv_inputs_kernel<TT, 1, 32><<<blocks(32), 256, 0, s>>>(a);       \
    else if (DP <= 32) wkv_inputs_kernel<TT, 4, 8><<<blocks(8), 256, 0, s>>>(a);   \
    else if (DP <= 64) wkv_inputs_kernel<TT, 4, 16><<<blocks(16), 256, 0, s>>>(a); \
    else wkv_inputs_kernel<TT, 4, 32><<<blocks(32), 256, 0, s>>>(a);           \
  } while (0)
  if (dtype == 0) B200_WI(__nv_bfloat16);
  else B200_WI(float);
#undef B200_WI
  return static_cast<int>(cudaGetLastError());
}

// Time mixing over the portions of a step (nd single tokens, then np portions by cu_q).
B200_API int b200_wkv_scan(const float* r, const float* k, const float* g, const float* v,
                           const float* now, float* out, float* matrix, const long long* positions,
                           const int* slots, int num_slots, const int* cu_q, int N, int D, int DP,
                           int VP, int nd, int np, void* stream) {
  if (nd + np <= 0) return 0;
  if (N <= 0 || D <= 0 || D > VP || (VP % 4) != 0) return -2;
  ScanArgs a{};
  a.q = r; a.k = k; a.g = g; a.v = v; a.s0 = now; a.out = out; a.matrix = matrix;
  a.positions = positions; a.slots = slots; a.num_slots = num_slots; a.cu_q = cu_q; a.G = N;
  a.N = N; a.D = D; a.V = D; a.VP = VP; a.nd = nd; a.np = np; a.ntaps = 1;
  return dispatch_scan<kWkv>(a, DP, nd + np, static_cast<cudaStream_t>(stream));
}

// out = tanh(x), n elements; dtype (of out): 0 bf16, 2 fp32.
B200_API int b200_tanh_rows(const float* x, void* out, long long n, int dtype, void* stream) {
  if (n <= 0) return 0;
  if (dtype != 0 && dtype != 2) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const unsigned int blocks = static_cast<unsigned int>((n + 255) / 256);
  if (dtype == 0)
    tanh_rows_kernel<__nv_bfloat16><<<blocks, 256, 0, s>>>(x, static_cast<__nv_bfloat16*>(out), n);
  else
    tanh_rows_kernel<float><<<blocks, 256, 0, s>>>(x, static_cast<float*>(out), n);
  return static_cast<int>(cudaGetLastError());
}

// One token of `nd` requests through time mixing, from the projections to the gated output: inner
// [nd, R] is the first step of the decay's projection (before its tanh), w2 [N D, R] the second's
// weights (R a multiple of 8, rows 16-byte aligned), gate the output gate's projection.  dtype: 0
// bf16, 2 fp32.  -20: not covered (very wide heads or ranks).
B200_API int b200_wkv_step(const void* r, const void* k, const void* v, const void* gate,
                           long long ld, const float* inner, long long ldi, int R, const void* w2,
                           const float* base, const float* bonus, const float* norm, float* matrix,
                           const long long* positions, const int* slots, int num_slots, void* out,
                           long long ldo, float eps, int nd, int N, int D, int DP, int dtype,
                           void* stream) {
  if (nd <= 0) return 0;
  if (N <= 0 || D <= 0 || D > DP || R <= 0 || (R % 8) != 0 ||
      (reinterpret_cast<uintptr_t>(w2) & 15) != 0 || (dtype != 0 && dtype != 2))
    return -2;
  StepArgs a{};
  a.H = R; a.x[0] = r; a.x[1] = k; a.x[2] = v; a.gate = gate; a.ldg = ld; a.ld = ld; a.z = inner;
  a.ldz = ldi; a.w0 = w2; a.b0 = base; a.b1 = bonus; a.qscale = 1.0f; a.norm = norm; a.per_head = 1;
  a.matrix = matrix; a.positions = positions; a.slots = slots; a.num_slots = num_slots; a.out = out;
  a.ldo = ldo; a.eps = eps; a.scale = 1.0f; a.G = N; a.N = N; a.D = D; a.V = D;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == 0 ? dispatch_step<__nv_bfloat16, kWkv>(a, DP, nd, s)
                    : dispatch_step<float, kWkv>(a, DP, nd, s);
}
