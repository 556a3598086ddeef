// Kernels around a 32-bit residual stream whose norms come after the sums (sm_100a).
//
//   token_shift     h[t] = x[t] + (x[t - 1] - x[t]) * mu, per coordinate; the row before the
//                   first row of a request's portion comes from the state that earlier steps
//                   left with the request's cache blocks (zero in front of position 0)
//   post_norm       r = rms(alpha * x + y) * g with one gain g per norm, where y is a dense row
//                   or the sum of a token's routed-expert rows; optionally followed in the same
//                   pass by the depth-weighted average x' = sum_j w[j] * X_j + w[n] * r over the
//                   results X_j of the layers so far, and by the final norm of that row
//   sigmoid_gate    o = o * sigmoid(z), z a strided view of a wider projection
//
// and around one whose norms sit on the sublayers' outputs only:
//
//   start_rows      x = s * embedding row (+ a vector); optionally the norm in front of the first
//                   sublayer in the same pass
//   add_normed      x = x + norm(y) (+ a vector) with a layer norm or an RMS norm (weight, optional
//                   bias); optionally the norm of the new row in the same pass (the final one, or
//                   that in front of the next sublayer).  y is a dense row, or the weighted sum of
//                   a token's routed-expert rows plus a shared expert's row times its gate
//   act_mul_rows    h = act(g) * u of rows [g | u], any width
//   ungated_act     h = max(u, 0)^2 or GELU
//   head_gate       o = o * sigmoid(z) * s from rows whose heads are padded
//
// The residual stream, the statistics and the averages are fp32; LO is the type of the rows that
// feed matrix products (bf16, or fp32 when the whole model runs in 32-bit).  One CTA per row,
// vectors of V elements (4 where every row is 4-aligned, else 1).
#include "rows.cuh"

namespace b200 {
namespace residual {

// ---------------------------------------------------------------------------
struct ShiftArgs {
  const float* x;          // [T, H]
  const float* mu;         // [H]
  const float* state;      // [num_blocks, H] last row written into every cache block, or null
  const int* block_tables; // [B, max_blocks]
  const long long* positions;
  const int* cu_q;         // [num_prefills + 1] relative to token num_decodes, or null
  void* out;               // [T, H]
  int T, H, num_decodes, num_prefills, max_blocks, block_size, num_blocks;
};

template <typename LO, int V>
__global__ void __launch_bounds__(256) token_shift_kernel(const ShiftArgs a) {
  const int t = blockIdx.x;
  const float* prev = nullptr;             // null: zeros
  const TokenPlace pl = token_place(t, a.num_decodes, a.num_prefills, a.cu_q);
  if (!pl.first) {
    prev = a.x + static_cast<long long>(t - 1) * a.H;
  } else if (a.state != nullptr && pl.req >= 0) {
    const long long pos = a.positions[t];
    if (pos > 0) {
      const long long bi = (pos - 1) / a.block_size;
      if (bi < a.max_blocks) {
        const int blk = a.block_tables[static_cast<long long>(pl.req) * a.max_blocks + bi];
        if (blk >= 0 && blk < a.num_blocks) prev = a.state + static_cast<long long>(blk) * a.H;
      }
    }
  }
  const float* x = a.x + static_cast<long long>(t) * a.H;
  LO* out = static_cast<LO*>(a.out) + static_cast<long long>(t) * a.H;
  for (int c = threadIdx.x * V; c < a.H; c += blockDim.x * V) {
    float xv[V], m[V], pv[V], o[V];
    ldv<V>(x + c, xv);
    ldv<V>(a.mu + c, m);
    if (prev != nullptr) {
      ldv<V>(prev + c, pv);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) pv[i] = 0.0f;
    }
#pragma unroll
    for (int i = 0; i < V; ++i) o[i] = xv[i] + (pv[i] - xv[i]) * m[i];
    stv<V>(out + c, o);
  }
}

// ---------------------------------------------------------------------------
struct PostNormArgs {
  const float* x;        // [T, H] residual stream
  const void* y;         // dense: [T, ldy]; routed: expert-sorted rows [cap, ldy]
  const int* pos_of;     // routed: [T, k] row of every (token, slot) pair (-1: none), else null
  const float* gain;     // scalar
  const float* hist;     // results of earlier layers: [n][T, H], hist_stride apart, or null
  const float* w;        // [n + 1] average weights (with hist)
  const float* fgain;    // final norm's scalar gain, or null
  float* res;            // [T, H] the norm's result, or null
  float* xo;             // [T, H] the average (with hist), or null
  void* lo;              // [T, H] LO copy: final-normed average, else the last fp32 result
  long long ldy, hist_stride;
  int T, H, k, n;
  float alpha, eps;
};

template <typename Y, typename LO, int V>
__global__ void __launch_bounds__(512) post_norm_kernel(const PostNormArgs a) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  float* z = sm;                 // [H]
  float* acc = sm + a.H;         // [H] partial average (with hist)
  const int t = blockIdx.x;
  const long long row = static_cast<long long>(t) * a.H;
  const Y* y = static_cast<const Y*>(a.y);
  float ss = 0.0f;
  for (int c = threadIdx.x * V; c < a.H; c += blockDim.x * V) {
    float xv[V], yv[V];
    ldv<V>(a.x + row + c, xv);
    if (a.pos_of == nullptr) {
      ldv<V>(y + static_cast<long long>(t) * a.ldy + c, yv);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) yv[i] = 0.0f;
      for (int s = 0; s < a.k; ++s) {
        const int p = a.pos_of[static_cast<long long>(t) * a.k + s];
        if (p < 0) continue;
        float f[V];
        ldv<V>(y + static_cast<long long>(p) * a.ldy + c, f);
#pragma unroll
        for (int i = 0; i < V; ++i) yv[i] += f[i];
      }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) {
      xv[i] = a.alpha * xv[i] + yv[i];
      ss += xv[i] * xv[i];
    }
    stv<V>(z + c, xv);
    if (a.hist != nullptr) {
      // the earlier results do not depend on this norm: read them while the row is in flight
      float s[V];
#pragma unroll
      for (int i = 0; i < V; ++i) s[i] = 0.0f;
      const float* hp = a.hist + row + c;
      int j = 0;
      for (; j + 4 <= a.n; j += 4) {
        float f0[V], f1[V], f2[V], f3[V];
        ldv<V>(hp + (j + 0) * a.hist_stride, f0);
        ldv<V>(hp + (j + 1) * a.hist_stride, f1);
        ldv<V>(hp + (j + 2) * a.hist_stride, f2);
        ldv<V>(hp + (j + 3) * a.hist_stride, f3);
        const float w0 = a.w[j], w1 = a.w[j + 1], w2 = a.w[j + 2], w3 = a.w[j + 3];
#pragma unroll
        for (int i = 0; i < V; ++i) s[i] += w0 * f0[i] + w1 * f1[i] + w2 * f2[i] + w3 * f3[i];
      }
      for (; j < a.n; ++j) {
        float f[V];
        ldv<V>(hp + j * a.hist_stride, f);
#pragma unroll
        for (int i = 0; i < V; ++i) s[i] += a.w[j] * f[i];
      }
      stv<V>(acc + c, s);
    }
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / static_cast<float>(a.H) + a.eps) * a.gain[0];
  LO* lo = static_cast<LO*>(a.lo);
  float ss2 = 0.0f;
  for (int c = threadIdx.x * V; c < a.H; c += blockDim.x * V) {
    float r[V];
    ldv<V>(z + c, r);
#pragma unroll
    for (int i = 0; i < V; ++i) r[i] *= inv;
    if (a.res != nullptr) stv<V>(a.res + row + c, r);
    if (a.hist != nullptr) {
      float s[V];
      ldv<V>(acc + c, s);
      const float wn = a.w[a.n];
#pragma unroll
      for (int i = 0; i < V; ++i) r[i] = s[i] + wn * r[i];
      if (a.xo != nullptr) stv<V>(a.xo + row + c, r);
    }
    if (lo != nullptr) {
      if (a.fgain == nullptr) {
        stv<V>(lo + row + c, r);
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) ss2 += r[i] * r[i];
        stv<V>(z + c, r);
      }
    }
  }
  if (lo == nullptr || a.fgain == nullptr) return;
  ss2 = block_sum(ss2, red);
  const float inv2 = 1.0f / sqrtf(ss2 / static_cast<float>(a.H) + a.eps) * a.fgain[0];
  for (int c = threadIdx.x * V; c < a.H; c += blockDim.x * V) {
    float r[V];
    ldv<V>(z + c, r);
#pragma unroll
    for (int i = 0; i < V; ++i) r[i] *= inv2;
    stv<V>(lo + row + c, r);
  }
}

// out[t, c] = o[t, c] * sigmoid(z[t, c])
template <typename T, int V>
__global__ void __launch_bounds__(256)
    sigmoid_gate_kernel(const T* o, long long ldo, const T* z, long long ldz, T* out,
                        long long ldout, long long rows, int D) {
  const int nv = D / V;
  const long long n = rows * nv;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < n;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long t = i / nv;
    const int c = static_cast<int>(i - t * nv) * V;
    float a[V], g[V];
    ldv<V>(o + t * ldo + c, a);
    ldv<V>(z + t * ldz + c, g);
#pragma unroll
    for (int k = 0; k < V; ++k) a[k] = a[k] / (1.0f + expf(-g[k]));
    stv<V>(out + t * ldout + c, a);
  }
}

// ---------------------------------------------------------------------------
struct StartArgs {
  const void* e;         // [T, lde] embedding rows
  const float* step;     // [H] vector added to every row, or null
  const float* w;        // [H] weight of the norm of the new row, or null
  float* x;              // [T, H]
  void* lo;              // [T, H] copy of x, or its norm
  long long lde;
  int H;
  float scale, eps;
};

template <typename T, int V>
__global__ void __launch_bounds__(512) start_rows_kernel(const StartArgs a) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const T* e = static_cast<const T*>(a.e) + t * a.lde;
  float* x = a.x + t * a.H;
  T* lo = static_cast<T*>(a.lo) + t * a.H;
  float ss = 0.0f;
  for (int c = threadIdx.x * V; c < a.H; c += blockDim.x * V) {
    float f[V];
    ldv<V>(e + c, f);
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] *= a.scale;
    if (a.step != nullptr) {
      float s[V];
      ldv<V>(a.step + c, s);
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] += s[i];
    }
    stv<V>(x + c, f);
    if (a.w == nullptr) stv<V>(lo + c, f);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += f[i] * f[i];
  }
  if (a.w == nullptr) return;
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / static_cast<float>(a.H) + a.eps);
  for (int c = threadIdx.x * V; c < a.H; c += blockDim.x * V) {   // what this thread wrote
    float f[V], w[V];
    ldv<V>(x + c, f);
    ldv<V>(a.w + c, w);
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] *= inv * w[i];
    stv<V>(lo + c, f);
  }
}

struct AddNormArgs {
  const float* x;        // [T, H] residual stream
  const void* y;         // [T, ldy] sublayer output; routed: expert-sorted rows [cap, ldy]
  const int* pos_of;     // routed: [T, k] row of every (token, slot) pair (-1: none), else null
  const float* row_w;    // routed: [T, k] weights
  const void* shared;    // routed: [T, ldsh] shared expert's rows, or null
  const float* gate;     // routed: logit of the shared expert's gate, one per ldg (null: no gate)
  const float* step;     // [H] vector added to the sum, or null
  const float* w;        // [H] norm weight
  const float* b;        // [H] norm bias, or null
  const float* fw;       // [H] final norm's weight, or null
  const float* fb;       // [H] final norm's bias, or null
  float* xo;             // [T, H] the sum (may be x), or null
  void* lo;              // [T, H] LO copy: of the sum, or of its final norm times fscale
  long long ldy, ldsh, ldg;
  int k;
  int T, H, centred;     // centred: layer norm (mean taken off), else RMS norm
  float eps, fscale;
};

// 1 / root of the mean square of z (minus its mean if `centred`); returns the mean in `mean`.
template <int V>
__device__ __forceinline__ float row_stats(const float* z, float sum, int H, int centred, float eps,
                                           float* red, float& mean) {
  mean = centred ? block_sum(sum, red) / static_cast<float>(H) : 0.0f;
  float ss = 0.0f;
  for (int c = threadIdx.x * V; c < H; c += blockDim.x * V) {
    float f[V];
    ldv<V>(z + c, f);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += (f[i] - mean) * (f[i] - mean);
  }
  ss = block_sum(ss, red);
  return 1.0f / sqrtf(ss / static_cast<float>(H) + eps);
}

template <typename T, int V, bool kRouted>
__global__ void __launch_bounds__(512) add_normed_kernel(const AddNormArgs a) {
  extern __shared__ float z[];       // [H]; every thread reads back only what it wrote
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const long long row = t * a.H;
  const T* y = static_cast<const T*>(a.y) + (kRouted ? 0 : t * a.ldy);
  float gate = 1.0f;
  if (kRouted && a.gate != nullptr) gate = 1.0f / (1.0f + expf(-a.gate[t * a.ldg]));
  float sum = 0.0f;
  for (int c = threadIdx.x * V; c < a.H; c += blockDim.x * V) {
    float f[V];
    if constexpr (kRouted) {
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] = 0.0f;
      for (int s = 0; s < a.k; ++s) {
        const int p = a.pos_of[t * a.k + s];
        if (p < 0) continue;
        const float w = a.row_w[t * a.k + s];
        float e[V];
        ldv<V>(y + static_cast<long long>(p) * a.ldy + c, e);
#pragma unroll
        for (int i = 0; i < V; ++i) f[i] += w * e[i];
      }
      if (a.shared != nullptr) {
        float e[V];
        ldv<V>(static_cast<const T*>(a.shared) + t * a.ldsh + c, e);
#pragma unroll
        for (int i = 0; i < V; ++i) f[i] += gate * e[i];
      }
    } else {
      ldv<V>(y + c, f);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) sum += f[i];
    stv<V>(z + c, f);
  }
  float mean;
  const float inv = row_stats<V>(z, sum, a.H, a.centred, a.eps, red, mean);
  T* lo = static_cast<T*>(a.lo) + row;
  sum = 0.0f;
  for (int c = threadIdx.x * V; c < a.H; c += blockDim.x * V) {
    float f[V], x[V], w[V], b[V];
    ldv<V>(z + c, f);
    ldv<V>(a.x + row + c, x);
    ldv<V>(a.w + c, w);
    if (a.b != nullptr) {
      ldv<V>(a.b + c, b);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) b[i] = 0.0f;
    }
#pragma unroll
    for (int i = 0; i < V; ++i) {
      x[i] += (f[i] - mean) * inv * w[i] + b[i];
    }
    if (a.step != nullptr) {
      ldv<V>(a.step + c, b);
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] += b[i];
    }
#pragma unroll
    for (int i = 0; i < V; ++i) sum += x[i];
    if (a.xo != nullptr) stv<V>(a.xo + row + c, x);
    if (a.fw == nullptr) stv<V>(lo + c, x);
    else stv<V>(z + c, x);
  }
  if (a.fw == nullptr) return;
  const float inv2 = row_stats<V>(z, sum, a.H, a.centred, a.eps, red, mean);
  for (int c = threadIdx.x * V; c < a.H; c += blockDim.x * V) {
    float f[V], w[V], b[V];
    ldv<V>(z + c, f);
    ldv<V>(a.fw + c, w);
    if (a.fb != nullptr) {
      ldv<V>(a.fb + c, b);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) b[i] = 0.0f;
    }
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = ((f[i] - mean) * inv2 * w[i] + b[i]) * a.fscale;
    stv<V>(lo + c, f);
  }
}

// The same for rows of whole vectors that fit the threads' registers, NI vectors each: the residual
// row is on its way while the sublayer's is summed, two expert rows are in flight at a time,
// and little but the sums goes through shared memory.
constexpr int kMaxSlots = 32;      // expert rows per token

template <typename T, int V, int NI, bool kRouted>
__global__ void __launch_bounds__(NI == 1 ? 1024 : 512) add_normed_reg_kernel(const AddNormArgs a) {
  __shared__ float red[32];
  __shared__ int s_pos[kMaxSlots];
  __shared__ float s_w[kMaxSlots];
  const long long t = blockIdx.x;
  const long long row = t * a.H;
  const int c0 = threadIdx.x * V, pitch = blockDim.x * V;
  const T* y = static_cast<const T*>(a.y) + (kRouted ? 0 : t * a.ldy);
  if (kRouted && threadIdx.x < a.k) {
    s_pos[threadIdx.x] = a.pos_of[t * a.k + threadIdx.x];
    s_w[threadIdx.x] = a.row_w[t * a.k + threadIdx.x];
  }
  float f[NI][V], x[NI][V];
#pragma unroll
  for (int n = 0; n < NI; ++n) {
    const int c = c0 + n * pitch;
#pragma unroll
    for (int i = 0; i < V; ++i) f[n][i] = x[n][i] = 0.0f;
    if (c >= a.H) continue;
    if constexpr (!kRouted) ldv<V>(y + c, f[n]);
    ldv<V>(a.x + row + c, x[n]);
  }
  if constexpr (kRouted) {
    // rows 0 .. k - 1 of the experts, row k the shared one
    const int rows = a.k + (a.shared != nullptr ? 1 : 0);
    const float gate = a.gate != nullptr ? 1.0f / (1.0f + expf(-a.gate[t * a.ldg])) : 1.0f;
    __syncthreads();
    auto place = [&](int s, const T*& e, float& w) {
      e = nullptr;
      w = 0.0f;
      if (s < a.k) {
        if (s_pos[s] >= 0) e = y + static_cast<long long>(s_pos[s]) * a.ldy;
        w = s_w[s];
      } else if (s < rows) {
        e = static_cast<const T*>(a.shared) + t * a.ldsh;
        w = gate;
      }
    };
    for (int s = 0; s < rows; s += 2) {
      const T *e0, *e1;
      float w0, w1;
      place(s, e0, w0);
      place(s + 1, e1, w1);
      float g0[NI][V], g1[NI][V];
#pragma unroll
      for (int n = 0; n < NI; ++n) {
        const int c = c0 + n * pitch;
#pragma unroll
        for (int i = 0; i < V; ++i) g0[n][i] = g1[n][i] = 0.0f;
        if (c < a.H && e0 != nullptr) ldv<V>(e0 + c, g0[n]);
        if (c < a.H && e1 != nullptr) ldv<V>(e1 + c, g1[n]);
      }
#pragma unroll
      for (int n = 0; n < NI; ++n)
#pragma unroll
        for (int i = 0; i < V; ++i) f[n][i] += w0 * g0[n][i] + w1 * g1[n][i];
    }
  }
  // mean (layer norm) and 1 / root of the mean square of the row in v
  auto stats = [&](const float (&v)[NI][V], float& mean) {
    mean = 0.0f;
    if (a.centred) {
      float sum = 0.0f;
#pragma unroll
      for (int n = 0; n < NI; ++n)
#pragma unroll
        for (int i = 0; i < V; ++i) sum += v[n][i];
      mean = block_sum(sum, red) / static_cast<float>(a.H);
    }
    float ss = 0.0f;
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      if (c0 + n * pitch >= a.H) continue;
#pragma unroll
      for (int i = 0; i < V; ++i) ss += (v[n][i] - mean) * (v[n][i] - mean);
    }
    return 1.0f / sqrtf(block_sum(ss, red) / static_cast<float>(a.H) + a.eps);
  };
  float mean;
  const float inv = stats(f, mean);
  T* lo = static_cast<T*>(a.lo) + row;
#pragma unroll
  for (int n = 0; n < NI; ++n) {
    const int c = c0 + n * pitch;
    if (c >= a.H) continue;
    float w[V], b[V];
    ldv<V>(a.w + c, w);
#pragma unroll
    for (int i = 0; i < V; ++i) x[n][i] += (f[n][i] - mean) * inv * w[i];
    if (a.b != nullptr) {
      ldv<V>(a.b + c, b);
#pragma unroll
      for (int i = 0; i < V; ++i) x[n][i] += b[i];
    }
    if (a.step != nullptr) {
      ldv<V>(a.step + c, b);
#pragma unroll
      for (int i = 0; i < V; ++i) x[n][i] += b[i];
    }
    if (a.xo != nullptr) stv<V>(a.xo + row + c, x[n]);
    if (a.fw == nullptr) stv<V>(lo + c, x[n]);
  }
  if (a.fw == nullptr) return;
  const float inv2 = stats(x, mean);
#pragma unroll
  for (int n = 0; n < NI; ++n) {
    const int c = c0 + n * pitch;
    if (c >= a.H) continue;
    float o[V], w[V], b[V] = {};
    ldv<V>(a.fw + c, w);
    if (a.fb != nullptr) ldv<V>(a.fb + c, b);
#pragma unroll
    for (int i = 0; i < V; ++i) o[i] = ((x[n][i] - mean) * inv2 * w[i] + b[i]) * a.fscale;
    stv<V>(lo + c, o);
  }
}

// out[t, h * D + c] = o[t, h * DC + c] * sigmoid(z[t, h * D + c]) * scale
template <typename T, int V>
__global__ void __launch_bounds__(512)
    head_gate_kernel(const T* o, int DC, const T* z, long long ldz, float scale, T* out,
                     long long ldout, int N, int D) {
  const long long t = blockIdx.x;
  const int nv = N * D / V;
  for (int i = threadIdx.x; i < nv; i += blockDim.x) {
    const int e = i * V;
    const int h = e / D, c = e - h * D;
    float a[V], g[V];
    ldv<V>(o + (t * N + h) * DC + c, a);
    ldv<V>(z + t * ldz + e, g);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      if constexpr (sizeof(T) == 2) a[k] = __fdividef(a[k] * scale, 1.0f + __expf(-g[k]));
      else a[k] = a[k] * scale / (1.0f + expf(-g[k]));
    }
    stv<V>(out + t * ldout + e, a);
  }
}

// activations by the codes of the GEMM epilogues (2 SiLU and 11 GELU-tanh, gated; 9 squared ReLU and
// 10 GELU); 32-bit models take the exact tanh
template <typename T, int ACT>
__device__ __forceinline__ float act_of(float x) {
  if constexpr (ACT == 2) return x / (1.0f + expf(-x));
  else if constexpr (ACT == 9) return relu2_f(x);
  else if constexpr (ACT == 10) return gelu_f(x);
  else if constexpr (sizeof(T) == 2) return gelu_tanh_f(x);
  else return 0.5f * x * (1.0f + tanhf(0.79788456080286536f * fmaf(0.044715f * x * x, x, x)));
}

template <typename T, int V, int ACT>
__global__ void __launch_bounds__(256)
    act_mul_rows_kernel(const T* x, long long ldx, T* out, long long ldo, int D) {
  const T* g = x + blockIdx.x * ldx;
  for (int c = threadIdx.x * V; c < D; c += blockDim.x * V) {
    float a[V], b[V];
    ldv<V>(g + c, a);
    ldv<V>(g + D + c, b);
#pragma unroll
    for (int i = 0; i < V; ++i) a[i] = act_of<T, ACT>(a[i]) * b[i];
    stv<V>(out + blockIdx.x * ldo + c, a);
  }
}

// out[t, c] = act(x[t, c]); may run in place
template <typename T, int V, int ACT>
__global__ void __launch_bounds__(256)
    ungated_act_kernel(const T* x, long long ldx, T* out, long long ldo, long long rows, int D) {
  const int nv = D / V;
  const long long n = rows * nv;
  for (long long i = blockIdx.x * static_cast<long long>(blockDim.x) + threadIdx.x; i < n;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long t = i / nv;
    const int c = static_cast<int>(i - t * nv) * V;
    float f[V];
    ldv<V>(x + t * ldx + c, f);
#pragma unroll
    for (int k = 0; k < V; ++k) f[k] = act_of<T, ACT>(f[k]);
    stv<V>(out + t * ldo + c, f);
  }
}

template <typename Y, typename LO, int V>
static int launch_post_norm(const PostNormArgs& a, cudaStream_t s) {
  const size_t smem = static_cast<size_t>(a.hist != nullptr ? 2 : 1) * a.H * sizeof(float);
  if (smem > 200 * 1024) return -2;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(post_norm_kernel<Y, LO, V>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  // few rows: more threads per row, so that a row's loads are in flight together
  const int threads = row_threads(a.H, V, a.T < 2 * sm_count() ? 512 : 256);
  post_norm_kernel<Y, LO, V><<<a.T, threads, smem, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int V, bool kRouted>
static int launch_add_normed_as(const AddNormArgs& a, cudaStream_t s) {
  // few rows: more threads per row, so that a row's loads are in flight together
  const bool few = a.T < 2 * sm_count();
  const int most = few ? 512 : 256;
  // 16-byte loads of the experts' 16-bit rows, of the fp32 row otherwise
  constexpr int R = kRouted ? 8 : 4;
  const int nvec = a.H / R;
  if (V == 4 && (a.H % R) == 0 && nvec <= 2048 && a.k <= kMaxSlots && a.ldy % R == 0 &&
      a.ldsh % R == 0) {
    const int ni = few && nvec <= 1024 ? 1 : (nvec <= 1024 ? 2 : 4);
    const int th = row_threads((nvec + ni - 1) / ni, 1, 1024);
    if (ni == 1) add_normed_reg_kernel<T, R, 1, kRouted><<<a.T, th, 0, s>>>(a);
    else if (ni == 2) add_normed_reg_kernel<T, R, 2, kRouted><<<a.T, th, 0, s>>>(a);
    else add_normed_reg_kernel<T, R, 4, kRouted><<<a.T, th, 0, s>>>(a);
    return static_cast<int>(cudaGetLastError());
  }
  const size_t smem = static_cast<size_t>(a.H) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(add_normed_kernel<T, V, kRouted>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  const int threads = row_threads(a.H, V, most);
  add_normed_kernel<T, V, kRouted><<<a.T, threads, smem, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}
template <typename T, int V>
static int launch_add_normed(const AddNormArgs& a, cudaStream_t s) {
  return a.pos_of != nullptr ? launch_add_normed_as<T, V, true>(a, s)
                             : launch_add_normed_as<T, V, false>(a, s);
}

}  // namespace residual
}  // namespace b200

using namespace b200;
using namespace b200::residual;

// out_dtype: 0 bf16, 2 fp32.  state / block_tables null: every portion starts from zeros.
B200_API int b200_token_shift(const float* x, const float* mu, const float* state,
                              const int* block_tables, const long long* positions, const int* cu_q,
                              void* out, int T, int H, int num_decodes, int num_prefills,
                              int max_blocks, int block_size, int num_blocks, int out_dtype,
                              void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || block_size <= 0 || (out_dtype != 0 && out_dtype != 2)) return -2;
  ShiftArgs a;
  a.x = x; a.mu = mu; a.state = block_tables ? state : nullptr; a.block_tables = block_tables;
  a.positions = positions; a.cu_q = cu_q; a.out = out; a.T = T; a.H = H;
  a.num_decodes = num_decodes; a.num_prefills = num_prefills; a.max_blocks = max_blocks;
  a.block_size = block_size; a.num_blocks = num_blocks;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool v4 = (H % 4) == 0 && aligned(x, 16) && aligned(mu, 16) && aligned(state, 16) &&
                  aligned(out, 16);
  const int th = row_threads(H, v4 ? 4 : 1, 256);
  if (out_dtype == 0) {
    if (v4) token_shift_kernel<__nv_bfloat16, 4><<<T, th, 0, s>>>(a);
    else token_shift_kernel<__nv_bfloat16, 1><<<T, th, 0, s>>>(a);
  } else {
    if (v4) token_shift_kernel<float, 4><<<T, th, 0, s>>>(a);
    else token_shift_kernel<float, 1><<<T, th, 0, s>>>(a);
  }
  return static_cast<int>(cudaGetLastError());
}

// dtype (of y and lo): 0 bf16, 2 fp32.  pos_of non-null: y holds expert-sorted rows, k per token.
// hist non-null: depth average over n earlier results.  The rows of res, xo and hist are H wide.
B200_API int b200_post_norm(const float* x, const void* y, long long ldy, const int* pos_of, int k,
                            const float* gain, float alpha, float eps, float* res,
                            const float* hist, long long hist_stride, int n, const float* w,
                            float* xo, const float* fgain, void* lo, int T, int H, int dtype,
                            void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || (dtype != 0 && dtype != 2) || (hist != nullptr && (w == nullptr || n < 0)))
    return -2;
  PostNormArgs a;
  a.x = x; a.y = y; a.ldy = ldy; a.pos_of = pos_of; a.k = k; a.gain = gain; a.alpha = alpha;
  a.eps = eps; a.res = res; a.hist = hist; a.hist_stride = hist_stride; a.n = n; a.w = w;
  a.xo = xo; a.fgain = fgain; a.lo = lo; a.T = T; a.H = H;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool v4 = (H % 4) == 0 && (ldy % 4) == 0 && (hist_stride % 4) == 0 && aligned(x, 16) &&
                  aligned(y, 16) && aligned(res, 16) && aligned(hist, 16) && aligned(xo, 16) &&
                  aligned(lo, 16);
  if (dtype == 0)
    return v4 ? launch_post_norm<__nv_bfloat16, __nv_bfloat16, 4>(a, s)
              : launch_post_norm<__nv_bfloat16, __nv_bfloat16, 1>(a, s);
  return v4 ? launch_post_norm<float, float, 4>(a, s) : launch_post_norm<float, float, 1>(a, s);
}

B200_API int b200_sigmoid_gate(const void* o, long long ldo, const void* z, long long ldz,
                               void* out, long long ldout, int T, int D, int dtype, void* stream) {
  if (T <= 0 || D <= 0) return 0;
  if (dtype != 0 && dtype != 2) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool v4 = (D % 4) == 0 && (ldo % 4) == 0 && (ldz % 4) == 0 && (ldout % 4) == 0 &&
                  aligned(o, 16) && aligned(z, dtype == 0 ? 8 : 16) && aligned(out, 16);
  const bool v8 = dtype == 0 && v4 && (D % 8) == 0 && (ldo % 8) == 0 && (ldz % 8) == 0 &&
                  (ldout % 8) == 0 && aligned(z, 16);
  const long long items = static_cast<long long>(T) * (v8 ? D / 8 : v4 ? D / 4 : D);
  long long blocks = (items + 255) / 256;
  const long long cap = static_cast<long long>(sm_count()) * 16;
  if (blocks > cap) blocks = cap;
  const int g = static_cast<int>(blocks);
  if (dtype == 0) {
    const __nv_bfloat16* po = static_cast<const __nv_bfloat16*>(o);
    const __nv_bfloat16* pz = static_cast<const __nv_bfloat16*>(z);
    __nv_bfloat16* pq = static_cast<__nv_bfloat16*>(out);
    if (v8) sigmoid_gate_kernel<__nv_bfloat16, 8><<<g, 256, 0, s>>>(po, ldo, pz, ldz, pq, ldout, T, D);
    else if (v4) sigmoid_gate_kernel<__nv_bfloat16, 4><<<g, 256, 0, s>>>(po, ldo, pz, ldz, pq, ldout, T, D);
    else sigmoid_gate_kernel<__nv_bfloat16, 1><<<g, 256, 0, s>>>(po, ldo, pz, ldz, pq, ldout, T, D);
  } else {
    const float* po = static_cast<const float*>(o);
    const float* pz = static_cast<const float*>(z);
    float* pq = static_cast<float*>(out);
    if (v4) sigmoid_gate_kernel<float, 4><<<g, 256, 0, s>>>(po, ldo, pz, ldz, pq, ldout, T, D);
    else sigmoid_gate_kernel<float, 1><<<g, 256, 0, s>>>(po, ldo, pz, ldz, pq, ldout, T, D);
  }
  return static_cast<int>(cudaGetLastError());
}

// x = scale * e (+ step) in fp32; lo in e's type: a copy of x, or with w its RMS norm times w.
// dtype (of e and lo): 0 bf16, 2 fp32.
B200_API int b200_start_rows(const void* e, long long lde, float scale, const float* step,
                             const float* w, float eps, float* x, void* lo, int T, int H, int dtype,
                             void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || (dtype != 0 && dtype != 2)) return -2;
  StartArgs a;
  a.e = e; a.step = step; a.w = w; a.x = x; a.lo = lo; a.lde = lde; a.H = H; a.scale = scale;
  a.eps = eps;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool v4 = (H % 4) == 0 && (lde % 4) == 0 && aligned(e, 16) && aligned(x, 16) &&
                  aligned(lo, 16) && aligned(step, 16) && aligned(w, 16);
  const int th = row_threads(H, v4 ? 4 : 1, T < 2 * sm_count() ? 512 : 256);
  if (dtype == 0) {
    if (v4) start_rows_kernel<__nv_bfloat16, 4><<<T, th, 0, s>>>(a);
    else start_rows_kernel<__nv_bfloat16, 1><<<T, th, 0, s>>>(a);
  } else {
    if (v4) start_rows_kernel<float, 4><<<T, th, 0, s>>>(a);
    else start_rows_kernel<float, 1><<<T, th, 0, s>>>(a);
  }
  return static_cast<int>(cudaGetLastError());
}

// xo = x + norm(y) * w + b (+ step); lo: the sum, or with fw (norm(sum) * fw + fb) * fscale.
// centred 1: layer norm, 0: RMS norm.  With pos_of [T, k]: y holds expert-sorted rows, and the row
// that is normalised is sum_s row_w[t, s] * y[pos_of[t, s]] + sigmoid(gate[t * ldg]) * shared[t].
// dtype (of y, shared and lo): 0 bf16, 2 fp32.
B200_API int b200_add_normed(const float* x, const void* y, long long ldy, const int* pos_of,
                             const float* row_w, int k, const void* shared, long long ldsh,
                             const float* gate, long long ldg, const float* step, const float* w,
                             const float* b, int centred, float eps, float* xo, const float* fw,
                             const float* fb, float fscale, void* lo, int T, int H, int dtype,
                             void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || (dtype != 0 && dtype != 2) || lo == nullptr ||
      (pos_of != nullptr && (row_w == nullptr || k <= 0)))
    return -2;
  AddNormArgs a;
  a.x = x; a.y = y; a.w = w; a.b = b; a.fw = fw; a.fb = fb; a.xo = xo; a.lo = lo; a.ldy = ldy;
  a.T = T; a.H = H; a.centred = centred; a.eps = eps; a.fscale = fscale; a.pos_of = pos_of;
  a.row_w = row_w; a.k = k; a.shared = shared; a.ldsh = ldsh; a.gate = gate; a.ldg = ldg;
  a.step = step;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool v4 = (H % 4) == 0 && (ldy % 4) == 0 && (ldsh % 4) == 0 && aligned(x, 16) &&
                  aligned(y, 16) && aligned(shared, 16) && aligned(step, 16) && aligned(w, 16) &&
                  aligned(b, 16) && aligned(fw, 16) && aligned(fb, 16) && aligned(xo, 16) &&
                  aligned(lo, 16);
  if (dtype == 0)
    return v4 ? launch_add_normed<__nv_bfloat16, 4>(a, s) : launch_add_normed<__nv_bfloat16, 1>(a, s);
  return v4 ? launch_add_normed<float, 4>(a, s) : launch_add_normed<float, 1>(a, s);
}

// out [T, D] = act(x), in place if the pointers are equal; act 9: max(x, 0)^2, 10: GELU; dtype 0 bf16,
// 2 fp32.
B200_API int b200_ungated_act(const void* x, long long ldx, void* out, long long ldo, int T, int D,
                              int act, int dtype, void* stream) {
  if (T <= 0 || D <= 0) return 0;
  if ((dtype != 0 && dtype != 2) || (act != 9 && act != 10)) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool v4 = (D % 4) == 0 && (ldx % 4) == 0 && (ldo % 4) == 0 && aligned(x, 16) &&
                  aligned(out, 16);
  const long long items = static_cast<long long>(T) * (v4 ? D / 4 : D);
  long long blocks = (items + 255) / 256;
  const long long cap = static_cast<long long>(sm_count()) * 16;
  const int g = static_cast<int>(blocks > cap ? cap : blocks);
#define B200_UA(TT, W, A)                                                                     \
  ungated_act_kernel<TT, W, A><<<g, 256, 0, s>>>(static_cast<const TT*>(x), ldx,             \
                                                 static_cast<TT*>(out), ldo, T, D)
#define B200_UA2(TT)                      \
  do {                                    \
    if (v4 && act == 9) B200_UA(TT, 4, 9); \
    else if (v4) B200_UA(TT, 4, 10);      \
    else if (act == 9) B200_UA(TT, 1, 9); \
    else B200_UA(TT, 1, 10);              \
  } while (0)
  if (dtype == 0) B200_UA2(__nv_bfloat16);
  else B200_UA2(float);
#undef B200_UA2
#undef B200_UA
  return static_cast<int>(cudaGetLastError());
}

// o [T, N, DC] -> out [T, N * D]: times sigmoid(z) and scale.
B200_API int b200_head_gate(const void* o, int DC, const void* z, long long ldz, float scale,
                            void* out, long long ldout, int T, int N, int D, int dtype,
                            void* stream) {
  if (T <= 0 || N <= 0 || D <= 0) return 0;
  if (DC < D || (dtype != 0 && dtype != 2)) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool v4 = (D % 4) == 0 && (DC % 4) == 0 && (ldz % 4) == 0 && (ldout % 4) == 0 &&
                  aligned(o, 16) && aligned(z, dtype == 0 ? 8 : 16) &&
                  aligned(out, dtype == 0 ? 8 : 16);
  const bool v8 = dtype == 0 && v4 && (D % 8) == 0 && (DC % 8) == 0 && (ldz % 8) == 0 &&
                  (ldout % 8) == 0 && aligned(z, 16) && aligned(out, 16);
  const int th = row_threads(N * D, v8 ? 8 : v4 ? 4 : 1, 512);
  if (dtype == 0) {
    const __nv_bfloat16* po = static_cast<const __nv_bfloat16*>(o);
    const __nv_bfloat16* pz = static_cast<const __nv_bfloat16*>(z);
    __nv_bfloat16* pq = static_cast<__nv_bfloat16*>(out);
    if (v8) head_gate_kernel<__nv_bfloat16, 8><<<T, th, 0, s>>>(po, DC, pz, ldz, scale, pq, ldout, N, D);
    else if (v4) head_gate_kernel<__nv_bfloat16, 4><<<T, th, 0, s>>>(po, DC, pz, ldz, scale, pq, ldout, N, D);
    else head_gate_kernel<__nv_bfloat16, 1><<<T, th, 0, s>>>(po, DC, pz, ldz, scale, pq, ldout, N, D);
  } else {
    const float* po = static_cast<const float*>(o);
    const float* pz = static_cast<const float*>(z);
    float* pq = static_cast<float*>(out);
    if (v4) head_gate_kernel<float, 4><<<T, th, 0, s>>>(po, DC, pz, ldz, scale, pq, ldout, N, D);
    else head_gate_kernel<float, 1><<<T, th, 0, s>>>(po, DC, pz, ldz, scale, pq, ldout, N, D);
  }
  return static_cast<int>(cudaGetLastError());
}

// out [T, D] = act(x[:, :D]) * x[:, D:]; act 2: SiLU, 11: GELU (tanh form); dtype 0 bf16, 2 fp32.
B200_API int b200_act_mul_rows(const void* x, long long ldx, void* out, long long ldo, int T, int D,
                               int act, int dtype, void* stream) {
  if (T <= 0 || D <= 0) return 0;
  if ((dtype != 0 && dtype != 2) || (act != 2 && act != 11)) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool v4 = (D % 4) == 0 && (ldx % 4) == 0 && (ldo % 4) == 0 && aligned(x, 16) &&
                  aligned(out, 16);
  const int th = row_threads(D, v4 ? 4 : 1, 256);
#define B200_AM(TT, W, A)                                                                 \
  act_mul_rows_kernel<TT, W, A><<<T, th, 0, s>>>(static_cast<const TT*>(x), ldx,          \
                                                 static_cast<TT*>(out), ldo, D)
#define B200_AM2(TT)                      \
  do {                                    \
    if (v4 && act == 2) B200_AM(TT, 4, 2); \
    else if (v4) B200_AM(TT, 4, 11);      \
    else if (act == 2) B200_AM(TT, 1, 2); \
    else B200_AM(TT, 1, 11);              \
  } while (0)
  if (dtype == 0) B200_AM2(__nv_bfloat16);
  else B200_AM2(float);
#undef B200_AM2
#undef B200_AM
  return static_cast<int>(cudaGetLastError());
}
