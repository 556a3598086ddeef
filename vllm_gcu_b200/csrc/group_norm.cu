// Kernels around a 32-bit residual stream with norms in front of the sublayers and a causal
// convolution behind the first of them (sm_100a).
//
//   add_group_norm  s = x + m * y, then h = s normalised in groups, times a weight: every one of
//                   `groups` consecutive parts of the row is divided by its own root mean square.  y
//                   is a dense row, or the weighted sum of a token's routed-expert rows plus a shared
//                   expert's row.  The leading single tokens of a step go on through the convolution
//                   (and the mixtures) below in the same pass.
//   input_conv      c = h + sum_j w[j] * h of (taps - 1 - j) tokens ago, per channel, over the
//                   portions of a step; optionally the mixtures c + (c' - c) * mu_m with the row c'
//                   of the token before, in place of c
//
// What the convolution needs of earlier steps lies in the request's state slot: a ring [back, H] in
// the model's type, row p % back holds h of position p (back = taps - 1, or taps with mixtures: c' is
// computed again from its inputs).  A ring's channel is read and written by one thread of a step, so
// neither slots nor rings need clearing or ordering: nothing is read in front of position 0.
//
// The residual stream, the statistics, the convolution and the mixtures are fp32; T is the type of
// the rows that feed matrix products (bf16, or fp32 when the whole model runs in 32-bit).
#include "rows.cuh"

namespace b200 {
namespace groupnorm {

constexpr int kMaxTaps = 8;
constexpr int kMaxSlots = 32;      // expert rows per token

struct ConvArgs {
  const float* w;          // [taps, H], the last tap meets the row itself
  const float* mu;         // [mixes, H] or null
  void* ring;              // [num_slots, back, H] or null
  const long long* positions;
  const int* slots;        // [requests]
  void* out;               // [T, H], or [mixes][T, H] mix_stride elements apart; row pitch ldo
  long long mix_stride, ldo;
  int taps, mixes, back, num_slots;
};

struct NormArgs {
  const float* x;          // [T, H] residual stream, or null: e
  const void* e;           // [T, lde] rows in the model's type (the embedding)
  const void* y;           // [T, ldy] sublayer output, or null; routed: expert-sorted rows
  const int* pos_of;       // routed: [T, k] row of every (token, slot) pair (-1: none), else null
  const float* row_w;      // routed: [T, k] weights
  const void* shared;      // routed: [T, ldsh] shared expert's rows, or null
  const float* gate;       // routed: logit of the shared expert's gate, one per ldg (null: no gate)
  const float* w;          // [H] norm weight
  float* xo;               // [T, H] the sum (may be x), or null
  void* lo;                // [T, H]
  long long lde, ldy, ldsh, ldg;
  int T, H, k, groups;
  int n1;                  // leading rows that go through the convolution
  float mult, eps;
  ConvArgs c;
};

// Partial sums of squares in shared memory: `run` neighbouring vectors (a power of two that divides
// a group's) per entry.
__host__ __device__ inline int run_length(int group_vectors) {
  int p = 1;
  while (p < 32 && group_vectors % (2 * p) == 0) p *= 2;
  return p;
}

template <typename T, int V, int NI, bool kRouted>
__global__ void __launch_bounds__(NI == 1 ? 1024 : 512) add_group_norm_kernel(const NormArgs a) {
  extern __shared__ float part[];            // [vectors / run], then [groups] where those are many
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
  float x[NI][V], f[NI][V];
#pragma unroll
  for (int n = 0; n < NI; ++n) {
    const int c = c0 + n * pitch;
#pragma unroll
    for (int i = 0; i < V; ++i) x[n][i] = f[n][i] = 0.0f;
    if (c >= a.H) continue;
    if (a.x != nullptr) ldv<V>(a.x + row + c, x[n]);
    else ldv<V>(static_cast<const T*>(a.e) + t * a.lde + c, x[n]);
    if (!kRouted && a.y != nullptr) ldv<V>(y + c, f[n]);
  }
  if constexpr (kRouted) {
    // rows 0 .. k - 1 of the experts, row k the shared one; two in flight at a time
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
  const int gv = a.H / a.groups / V, run = run_length(gv), per = gv / run;
#pragma unroll
  for (int n = 0; n < NI; ++n) {
    const int c = c0 + n * pitch;
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      x[n][i] += a.mult * f[n][i];
      ss += x[n][i] * x[n][i];
    }
    for (int o = 1; o < run; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (c >= a.H) continue;
    if (a.xo != nullptr) stv<V>(a.xo + row + c, x[n]);
    const int v = c / V;
    if (v % run == 0) part[v / run] = ss;
  }
  __syncthreads();
  constexpr int kDirect = 16;                // partial sums a thread adds up itself
  float* whole = part + a.H / V / run;
  if (per > kDirect) {
    for (int g = threadIdx.x >> 5; g < a.groups; g += blockDim.x >> 5) {
      float ss = 0.0f;
      for (int i = threadIdx.x & 31; i < per; i += 32) ss += part[g * per + i];
      ss = warp_sum(ss);
      if ((threadIdx.x & 31) == 0) whole[g] = ss;
    }
    __syncthreads();
  }
  const float width = static_cast<float>(a.H / a.groups);
  const ConvArgs& cv = a.c;
  const bool conv = t < a.n1;
  int pos = 0;
  T* ring = nullptr;
  if (conv) {
    const int slot = cv.slots[t];
    pos = static_cast<int>(cv.positions[t]);
    if (cv.ring != nullptr && slot >= 0 && slot < cv.num_slots)
      ring = static_cast<T*>(cv.ring) + static_cast<long long>(slot) * cv.back * a.H;
  }
#pragma unroll
  for (int n = 0; n < NI; ++n) {
    const int c = c0 + n * pitch;
    if (c >= a.H) continue;
    const int g = c / V / gv;
    float ss = 0.0f;
    if (per > kDirect) {
      ss = whole[g];
    } else {
      for (int i = 0; i < per; ++i) ss += part[g * per + i];
    }
    const float inv = 1.0f / sqrtf(ss / width + a.eps);
    float w[V], h[V];
    ldv<V>(a.w + c, w);
#pragma unroll
    for (int i = 0; i < V; ++i) h[i] = x[n][i] * inv * w[i];
    if (!conv) {
      stv<V>(static_cast<T*>(a.lo) + row + c, h);
      continue;
    }
    // what portions read back is the rounded row
    float now[V], before[V];
    ldv<V>(cv.w + static_cast<long long>(cv.taps - 1) * a.H + c, w);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      h[i] = round_like<T>(h[i]);
      now[i] = h[i] + h[i] * w[i];
      before[i] = 0.0f;
    }
    if (ring != nullptr) {
      for (int o = 1; o <= cv.back && pos - o >= 0; ++o) {
        float r[V];
        ldv<V>(ring + static_cast<long long>((pos - o) % cv.back) * a.H + c, r);
        if (cv.mu != nullptr) {
          // w: the tap that meets this row in the convolution of the token before
#pragma unroll
          for (int i = 0; i < V; ++i) before[i] += r[i] * w[i] + (o == 1 ? r[i] : 0.0f);
        }
        if (o < cv.taps) {
          ldv<V>(cv.w + static_cast<long long>(cv.taps - 1 - o) * a.H + c, w);
#pragma unroll
          for (int i = 0; i < V; ++i) now[i] += r[i] * w[i];
        }
      }
      stv<V>(ring + static_cast<long long>(pos % cv.back) * a.H + c, h);
    }
    T* out = static_cast<T*>(cv.out) + t * cv.ldo + c;
    if (cv.mu == nullptr) {
      stv<V>(out, now);
      continue;
    }
    for (int m = 0; m < cv.mixes; ++m) {
      float u[V], o[V];
      ldv<V>(cv.mu + static_cast<long long>(m) * a.H + c, u);
#pragma unroll
      for (int i = 0; i < V; ++i) o[i] = now[i] + (before[i] - now[i]) * u[i];
      stv<V>(out + m * cv.mix_stride, o);
    }
  }
}

// ---------------------------------------------------------------------------
constexpr int kStrip = 16;         // tokens a CTA walks; at least kMaxTaps: later strips of a
                                   // portion do not look in front of it

struct PortionArgs {
  const void* h;           // [T, H]
  const int* cu_q;         // [np + 1] relative to token nd, or null
  int H, nd, np;
  ConvArgs c;
};

// V neighbouring elements as they lie in memory
template <typename T, int V>
struct RawRow {
  T e[V];
};
template <>
struct __align__(16) RawRow<__nv_bfloat16, 8> {
  uint4 u;
};
template <>
struct __align__(16) RawRow<float, 4> {
  float4 u;
};
template <typename T, int V>
__device__ __forceinline__ RawRow<T, V> load_raw(const T* p) {
  return *reinterpret_cast<const RawRow<T, V>*>(p);
}
template <typename T, int V>
__device__ __forceinline__ void unpack_raw(const RawRow<T, V>& r, float (&f)[V]) {
  if constexpr (V == 8) {
    const uint32_t w[4] = {r.u.x, r.u.y, r.u.z, r.u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 p = unpack_bf16x2(w[i]);
      f[2 * i] = p.x;
      f[2 * i + 1] = p.y;
    }
  } else if constexpr (V == 4) {
    f[0] = r.u.x; f[1] = r.u.y; f[2] = r.u.z; f[3] = r.u.w;
  } else {
    f[0] = to_f32<T>(r.e[0]);
  }
}

// grid.x: at least the strips of all requests; grid.y: slabs of blockDim.x * V channels.
template <typename T, int V, int NT, bool kMixed>
__global__ void __launch_bounds__(256, NT <= 4 ? 2 : 1) input_conv_kernel(const PortionArgs a) {
  constexpr int kBatch = kMixed ? 4 : 8;     // rows in flight
  __shared__ int s_req, s_strip;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x, want = blockIdx.x;
    int found = -1, strip = 0, base = 0;
    const int requests = a.nd + a.np;
    for (int r0 = 0; r0 < requests && found < 0; r0 += 32) {
      const int r = r0 + lane;
      int n = 0;
      if (r < requests)
        n = r < a.nd ? 1 : (a.cu_q[r - a.nd + 1] - a.cu_q[r - a.nd] + kStrip - 1) / kStrip;
      int inc = n;
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, inc, d);
        if (lane >= d) inc += u;
      }
      const int start = base + inc - n;
      const unsigned int vote =
          __ballot_sync(0xffffffffu, n > 0 && want >= start && want < start + n);
      if (vote != 0u) {
        const int src = __ffs(vote) - 1;
        found = r0 + src;
        strip = want - __shfl_sync(0xffffffffu, start, src);
      }
      base += __shfl_sync(0xffffffffu, inc, 31);
    }
    if (lane == 0) {
      s_req = found;
      s_strip = strip;
    }
  }
  __syncthreads();
  const int req = s_req;
  if (req < 0) return;                       // surplus CTA
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= a.H) return;
  const int first = req < a.nd ? req : a.nd + a.cu_q[req - a.nd];
  const int count = req < a.nd ? 1 : a.cu_q[req - a.nd + 1] - a.cu_q[req - a.nd];
  const int i0 = s_strip * kStrip, i1 = min(count, i0 + kStrip);
  const ConvArgs& cv = a.c;
  const int p0 = static_cast<int>(cv.positions[first]);
  const int slot = cv.slots[req];
  T* ring = nullptr;
  if (cv.ring != nullptr && slot >= 0 && slot < cv.num_slots)
    ring = static_cast<T*>(cv.ring) + static_cast<long long>(slot) * cv.back * a.H + c;
  const T* h = static_cast<const T*>(a.h) + static_cast<long long>(first) * a.H + c;

  float w[NT][V];                            // [o]: tap that meets the row of o tokens ago
#pragma unroll
  for (int o = 0; o < NT; ++o) {
#pragma unroll
    for (int i = 0; i < V; ++i) w[o][i] = 0.0f;
    if (o < cv.taps) ldv<V>(cv.w + static_cast<long long>(cv.taps - 1 - o) * a.H + c, w[o]);
  }
  RawRow<T, V> past[NT];                     // [o]: row of o + 1 tokens ago, as it lies in memory
#pragma unroll
  for (int o = 0; o < NT; ++o) {
    past[o] = RawRow<T, V>{};
    if (o >= cv.back) continue;
    const int i = i0 - 1 - o;
    if (i >= 0) past[o] = load_raw<T, V>(h + static_cast<long long>(i) * a.H);
    else if (ring != nullptr && p0 + i >= 0)
      past[o] = load_raw<T, V>(ring + static_cast<long long>((p0 + i) % cv.back) * a.H);
  }
  // now[1 ..]: convolved rows of the batch; now[0]: the one in front of it
  float now[kBatch + 1][V];
  if (kMixed) {
#pragma unroll
    for (int o = 0; o < NT; ++o) {
      float f[V];
      unpack_raw<T, V>(past[o], f);
#pragma unroll
      for (int i = 0; i < V; ++i) now[kBatch][i] = (o == 0 ? f[i] : now[kBatch][i]) + w[o][i] * f[i];
    }
  }
  T* out = static_cast<T*>(cv.out) + static_cast<long long>(first) * cv.ldo + c;
#pragma unroll 1
  for (int b = i0; b < i1; b += kBatch) {
    RawRow<T, V> rows[kBatch];               // all rows of the batch in flight at once
#pragma unroll
    for (int u = 0; u < kBatch; ++u) {
      rows[u] = RawRow<T, V>{};
      if (b + u < i1) rows[u] = load_raw<T, V>(h + static_cast<long long>(b + u) * a.H);
    }
    if (kMixed) {
#pragma unroll
      for (int i = 0; i < V; ++i) now[0][i] = now[kBatch][i];
    }
#pragma unroll
    for (int u = 0; u < kBatch; ++u) {
      float* n = now[u + 1];
      float f[V];
      unpack_raw<T, V>(rows[u], f);
#pragma unroll
      for (int i = 0; i < V; ++i) n[i] = f[i] + w[0][i] * f[i];
#pragma unroll
      for (int o = 1; o < NT; ++o) {
        unpack_raw<T, V>(past[o - 1], f);
#pragma unroll
        for (int i = 0; i < V; ++i) n[i] += w[o][i] * f[i];
      }
#pragma unroll
      for (int o = NT - 1; o > 0; --o) past[o] = past[o - 1];
      past[0] = rows[u];
      if (!kMixed && b + u < i1) stv<V>(out + static_cast<long long>(b + u) * cv.ldo, now[u + 1]);
    }
    if (!kMixed) continue;
    for (int m = 0; m < cv.mixes; ++m) {
      float k[V];
      ldv<V>(cv.mu + static_cast<long long>(m) * a.H + c, k);
#pragma unroll
      for (int u = 0; u < kBatch; ++u) {
        if (b + u >= i1) break;
        float o[V];
#pragma unroll
        for (int i = 0; i < V; ++i) o[i] = now[u + 1][i] + (now[u][i] - now[u + 1][i]) * k[i];
        stv<V>(out + static_cast<long long>(b + u) * cv.ldo + m * cv.mix_stride, o);
      }
    }
  }
  // the portion's last rows -> ring, by the threads that have read it
  if (i0 > 0 || ring == nullptr) return;
  for (int i = max(0, count - cv.back); i < count; ++i) {
    float r[V];
    ldv<V>(h + static_cast<long long>(i) * a.H, r);
    stv<V>(ring + static_cast<long long>((p0 + i) % cv.back) * a.H, r);
  }
}

template <typename T, int V, int NI, bool kRouted>
static int launch_norm(const NormArgs& a, int threads, cudaStream_t s) {
  const int run = run_length(a.H / a.groups / V);
  const size_t smem = (static_cast<size_t>(a.H / V / run) + a.groups) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(add_group_norm_kernel<T, V, NI, kRouted>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  add_group_norm_kernel<T, V, NI, kRouted><<<a.T, threads, smem, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int V, bool kRouted>
static int dispatch_norm(const NormArgs& a, cudaStream_t s) {
  // few rows: more threads per row, so that a row's loads are in flight together
  const bool few = a.T < 2 * sm_count();
  const int vectors = a.H / V;
  if (few && vectors <= 1024) return launch_norm<T, V, 1, kRouted>(a, row_threads(vectors, 1, 1024), s);
  if (vectors <= 1024)
    return launch_norm<T, V, 2, kRouted>(a, row_threads((vectors + 1) / 2, 1, 512), s);
  if (vectors <= 2048)
    return launch_norm<T, V, 4, kRouted>(a, row_threads((vectors + 3) / 4, 1, 512), s);
  if constexpr (V == 4) {
    if (vectors <= 4096)
      return launch_norm<T, V, 8, kRouted>(a, row_threads((vectors + 7) / 8, 1, 512), s);
  } else if constexpr (V == 1) {
    if (vectors <= 8192)
      return launch_norm<T, V, 16, kRouted>(a, row_threads((vectors + 15) / 16, 1, 512), s);
  }
  return -20;
}

template <typename T>
static int dispatch_norm(const NormArgs& a, bool vec, cudaStream_t s) {
  constexpr int V = sizeof(T) == 2 ? 8 : 4;
  if (a.pos_of != nullptr)
    return vec ? dispatch_norm<T, V, true>(a, s) : dispatch_norm<T, 1, true>(a, s);
  return vec ? dispatch_norm<T, V, false>(a, s) : dispatch_norm<T, 1, false>(a, s);
}

static bool bad_conv(const ConvArgs& c) {
  return c.taps < 1 || c.taps > kMaxTaps || c.back != (c.mu != nullptr ? c.taps : c.taps - 1) ||
         (c.mu != nullptr && c.mixes < 1) || c.positions == nullptr || c.slots == nullptr ||
         c.out == nullptr;
}

}  // namespace groupnorm
}  // namespace b200

using namespace b200;
using namespace b200::groupnorm;

// xo = (x or e) + mult * y; h = xo normalised in groups, times w.  Rows from n1 on: lo = h; rows
// before: through the convolution to conv_out (mixes > 0: that many mixtures, mix_stride elements
// apart).  With pos_of [T, k]: y holds expert-sorted rows and is sum_s row_w[t, s] * y[pos_of[t, s]]
// + sigmoid(gate[t * ldg]) * shared[t] (gate null: 1).  dtype (of e, y, shared, lo, conv_out and the
// ring): 0 bf16, 2 fp32.  -20: a width the kernel does not cover (16384, or 8192 of an odd kind).
B200_API int b200_add_group_norm(const float* x, const void* e, long long lde, const void* y,
                                 long long ldy, float mult, const int* pos_of, const float* row_w,
                                 int k, const void* shared, long long ldsh, const float* gate,
                                 long long ldg, const float* w, int groups, float eps, float* xo,
                                 void* lo, const float* conv_w, int taps, const float* mu, int mixes,
                                 void* ring, int num_slots, const long long* positions,
                                 const int* slots, void* conv_out, long long mix_stride,
                                 long long conv_ld, int n1, int T, int H, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || groups <= 0 || H % groups != 0 || (dtype != 0 && dtype != 2) ||
      (x == nullptr) == (e == nullptr) || n1 < 0 || n1 > T || (n1 < T && lo == nullptr) ||
      (pos_of != nullptr && (row_w == nullptr || y == nullptr || k <= 0 || k > kMaxSlots)))
    return -2;
  NormArgs a;
  a.x = x; a.e = e; a.lde = lde; a.y = y; a.ldy = ldy; a.mult = mult; a.pos_of = pos_of;
  a.row_w = row_w; a.k = k; a.shared = shared; a.ldsh = ldsh; a.gate = gate; a.ldg = ldg; a.w = w;
  a.groups = groups; a.eps = eps; a.xo = xo; a.lo = lo; a.T = T; a.H = H; a.n1 = n1;
  a.c = ConvArgs{conv_w, mu, ring, positions, slots, conv_out, mix_stride, conv_ld, taps, mixes,
                 mu != nullptr ? taps : taps - 1, num_slots};
  if (n1 > 0 && bad_conv(a.c)) return -2;
  const int V = dtype == 0 ? 8 : 4;
  const bool vec = (H / groups) % V == 0 && (lde % V) == 0 && (ldy % V) == 0 && (ldsh % V) == 0 &&
                   (conv_ld % V) == 0 && (mix_stride % V) == 0 && aligned(x, 16) &&
                   aligned(e, 16) && aligned(y, 16) && aligned(shared, 16) && aligned(w, 16) &&
                   aligned(xo, 16) && aligned(lo, 16) && aligned(conv_w, 16) && aligned(mu, 16) &&
                   aligned(ring, 16) && aligned(conv_out, 16);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == 0 ? dispatch_norm<__nv_bfloat16>(a, vec, s) : dispatch_norm<float>(a, vec, s);
}

// The convolution over the portions of a step (nd single tokens, then np portions by cu_q); see
// above.  h [T, H]; rows of no request are left as they are.
B200_API int b200_input_conv(const void* h, const float* w, int taps, const float* mu, int mixes,
                             void* ring, int num_slots, const long long* positions,
                             const int* slots, const int* cu_q, void* out, long long mix_stride,
                             long long ldo, int T, int H, int nd, int np, int dtype, void* stream) {
  if (T <= 0 || nd + np <= 0) return 0;
  if (H <= 0 || (dtype != 0 && dtype != 2) || nd < 0 || np < 0 || (np > 0 && cu_q == nullptr))
    return -2;
  PortionArgs a;
  a.h = h; a.cu_q = cu_q; a.H = H; a.nd = nd; a.np = np;
  a.c = ConvArgs{w, mu, ring, positions, slots, out, mix_stride, ldo, taps, mixes,
                 mu != nullptr ? taps : taps - 1, num_slots};
  if (bad_conv(a.c)) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int V = dtype == 0 ? 8 : 4;
  const bool vec = (H % V) == 0 && (ldo % V) == 0 && (mix_stride % V) == 0 && aligned(h, 16) &&
                   aligned(w, 16) && aligned(mu, 16) && aligned(ring, 16) && aligned(out, 16);
  const int lanes = vec ? H / V : H;
  const int th = row_threads(lanes, 1, 256);
  // sum of ceil(n_r / kStrip) <= T / kStrip + requests
  const dim3 grid(T / kStrip + nd + np, (lanes + th - 1) / th);
#define B200_IC(TT, W)                                                    \
  do {                                                                    \
    if (taps <= 4 && mu == nullptr)                                       \
      input_conv_kernel<TT, W, 4, false><<<grid, th, 0, s>>>(a);          \
    else if (taps <= 4)                                                   \
      input_conv_kernel<TT, W, 4, true><<<grid, th, 0, s>>>(a);           \
    else if (mu == nullptr)                                               \
      input_conv_kernel<TT, W, 8, false><<<grid, th, 0, s>>>(a);          \
    else                                                                  \
      input_conv_kernel<TT, W, 8, true><<<grid, th, 0, s>>>(a);           \
  } while (0)
  if (dtype == 0) {
    if (vec) B200_IC(__nv_bfloat16, 8);
    else B200_IC(__nv_bfloat16, 1);
  } else {
    if (vec) B200_IC(float, 4);
    else B200_IC(float, 1);
  }
#undef B200_IC
  return static_cast<int>(cudaGetLastError());
}
