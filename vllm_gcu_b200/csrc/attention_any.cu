// Kernels of key / value attention outside the tensor-core layouts, and the kernel in front of it.
//
//   qk_norm_rope_cache  RMS norm of a query and of a key row over the whole projection (all heads
//                       at once), rotary positions on the first dimensions of every head, queries
//                       to a padded buffer, keys and values to the paged cache.  Values are a
//                       projection of their own or the keys as they were before the norm.
//   head_norm_cache     RMS norm of every query and key head over its own dimensions with one
//                       weight for all heads, no positions; queries to a padded buffer, keys and
//                       values (of another width, if so) to the paged cache.  One warp per head.
//   qkv_cache           what grouped attention needs of its projections in one pass: norm over the
//                       whole query and key rows, rotation (i with i + rot / 2), temperature of the
//                       queries by position, norm of every head's values, values mixed with those
//                       that an earlier layer has cached for the token; each optional
//   any_attention       causal paged attention for any head dimension and group size, fp32 or
//                       bf16 rows, optional sink, soft cap, chunks of positions, sliding window and
//                       distance bias: serves models that run in 32-bit and the shapes the tensor-core kernels do not cover.
//
// Cache layout as in attention.cu: [num_slots, kv_heads, DC] with DC >= D, zeros behind D.
#include "common.cuh"

namespace b200 {
namespace anyattn {

constexpr unsigned int kKernelId = 74;

struct PrepArgs {
  const void* q;             // [T, Hq * D] view, row pitch ldq
  const void* k;             // [T, Hkv * D]
  const void* v;             // [T, Hkv * D], or null: the keys before their norm
  const float* qw;           // [Hq * D] norm weights
  const float* kw;           // [Hkv * D]
  const float* sumsq;        // [T, 2] sums of squares of the whole q / k rows, or null: these rows
  const float* cos_sin;      // [positions, rot] cos | sin
  const long long* positions;
  const long long* slots;    // [T] (-1: no cache write)
  void* qo;                  // [T, Hq, DC]
  void* kc;                  // [num_slots, Hkv, DC]
  void* vc;
  long long ldq, ldk, ldv, num_slots, max_pos;
  int T, Hq, Hkv, D, DC, rot, q_all, k_all, is_neox;
  float eps;
  unsigned int* status;
};

// Normalised (and rotated) element c of head `h`: x is the projected row, inv its 1 / rms.
template <typename T>
__device__ __forceinline__ float rotated(const T* x, const float* w, float inv, int base, int c,
                                         int rot, int is_neox, const float* cs) {
  const float self = to_f32<T>(x[base + c]) * inv * w[base + c];
  if (c >= rot) return self;
  const int half = rot / 2;
  int i, mate;
  bool first;
  if (is_neox) {
    first = c < half;
    i = first ? c : c - half;
    mate = first ? c + half : c - half;
  } else {
    first = (c & 1) == 0;
    i = c >> 1;
    mate = c ^ 1;
  }
  const float other = to_f32<T>(x[base + mate]) * inv * w[base + mate];
  const float co = cs[i], si = cs[half + i];
  return first ? self * co - other * si : self * co + other * si;
}

template <typename T>
__global__ void __launch_bounds__(256) qk_norm_rope_cache_kernel(const PrepArgs a) {
  __shared__ float red[32];
  const int t = blockIdx.x;
  const T* q = static_cast<const T*>(a.q) + static_cast<long long>(t) * a.ldq;
  const T* k = static_cast<const T*>(a.k) + static_cast<long long>(t) * a.ldk;
  const int nq = a.Hq * a.D, nk = a.Hkv * a.D;
  float sq = 0.0f, sk = 0.0f;
  if (a.sumsq != nullptr) {
    sq = a.sumsq[2 * t];
    sk = a.sumsq[2 * t + 1];
  } else {
    for (int c = threadIdx.x; c < nq; c += blockDim.x) {
      const float f = to_f32<T>(q[c]);
      sq += f * f;
    }
    for (int c = threadIdx.x; c < nk; c += blockDim.x) {
      const float f = to_f32<T>(k[c]);
      sk += f * f;
    }
    sq = block_sum(sq, red);
    sk = block_sum(sk, red);
  }
  const float qi = 1.0f / sqrtf(sq / static_cast<float>(a.q_all) + a.eps);
  const float ki = 1.0f / sqrtf(sk / static_cast<float>(a.k_all) + a.eps);
  long long pos = a.positions[t];
  if (pos < 0 || pos >= a.max_pos) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId, static_cast<unsigned int>(t));
    pos = 0;
  }
  const float* cs = a.cos_sin + pos * a.rot;
  T* qo = static_cast<T*>(a.qo) + static_cast<long long>(t) * a.Hq * a.DC;
  for (int e = threadIdx.x; e < a.Hq * a.DC; e += blockDim.x) {
    const int h = e / a.DC, c = e - h * a.DC;
    qo[e] = from_f32<T>(c < a.D ? rotated<T>(q, a.qw, qi, h * a.D, c, a.rot, a.is_neox, cs) : 0.0f);
  }
  const long long slot = a.slots[t];
  if (slot < 0) return;
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId + 1, static_cast<unsigned int>(t));
    return;
  }
  const T* v = a.v != nullptr ? static_cast<const T*>(a.v) + static_cast<long long>(t) * a.ldv : k;
  T* kc = static_cast<T*>(a.kc) + slot * a.Hkv * a.DC;
  T* vc = static_cast<T*>(a.vc) + slot * a.Hkv * a.DC;
  for (int e = threadIdx.x; e < a.Hkv * a.DC; e += blockDim.x) {
    const int h = e / a.DC, c = e - h * a.DC;
    const bool in = c < a.D;
    kc[e] = from_f32<T>(in ? rotated<T>(k, a.kw, ki, h * a.D, c, a.rot, a.is_neox, cs) : 0.0f);
    vc[e] = in ? v[h * a.D + c] : from_f32<T>(0.0f);
  }
}

// The same for bf16 rows, two neighbouring elements per thread (D, DC and rot even, pairs of
// neighbours rotated together).
__global__ void __launch_bounds__(256) qk_norm_rope_cache_pairs_kernel(const PrepArgs a) {
  __shared__ float red[32];
  const int t = blockIdx.x;
  const __nv_bfloat16* q =
      static_cast<const __nv_bfloat16*>(a.q) + static_cast<long long>(t) * a.ldq;
  const __nv_bfloat16* k =
      static_cast<const __nv_bfloat16*>(a.k) + static_cast<long long>(t) * a.ldk;
  auto pair = [](const __nv_bfloat16* p, int i) {
    return unpack_bf16x2(reinterpret_cast<const uint32_t*>(p)[i]);
  };
  const int nq = a.Hq * a.D / 2, nk = a.Hkv * a.D / 2;
  float sq = 0.0f, sk = 0.0f;
  if (a.sumsq != nullptr) {
    sq = a.sumsq[2 * t];
    sk = a.sumsq[2 * t + 1];
  } else {
    for (int i = threadIdx.x; i < nq; i += blockDim.x) {
      const float2 f = pair(q, i);
      sq += f.x * f.x + f.y * f.y;
    }
    for (int i = threadIdx.x; i < nk; i += blockDim.x) {
      const float2 f = pair(k, i);
      sk += f.x * f.x + f.y * f.y;
    }
    sq = block_sum(sq, red);
    sk = block_sum(sk, red);
  }
  const float qi = 1.0f / sqrtf(sq / static_cast<float>(a.q_all) + a.eps);
  const float ki = 1.0f / sqrtf(sk / static_cast<float>(a.k_all) + a.eps);
  long long pos = a.positions[t];
  if (pos < 0 || pos >= a.max_pos) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId, static_cast<unsigned int>(t));
    pos = 0;
  }
  const float* cs = a.cos_sin + pos * a.rot;
  const int half = a.rot / 2, dp = a.D / 2, dcp = a.DC / 2;
  auto turned = [&](const __nv_bfloat16* x, const float* w, float inv, int i, int c) {
    const float2 f = pair(x, i);
    const float2 g = reinterpret_cast<const float2*>(w)[i];
    const float u = f.x * inv * g.x, v = f.y * inv * g.y;
    if (c >= half) return pack_bf16x2(u, v);
    const float co = cs[c], si = cs[half + c];
    return pack_bf16x2(u * co - v * si, v * co + u * si);
  };
  uint32_t* qo = reinterpret_cast<uint32_t*>(a.qo) + static_cast<long long>(t) * a.Hq * dcp;
  for (int e = threadIdx.x; e < a.Hq * dcp; e += blockDim.x) {
    const int h = e / dcp, c = e - h * dcp;
    qo[e] = c < dp ? turned(q, a.qw, qi, h * dp + c, c) : 0u;
  }
  const long long slot = a.slots[t];
  if (slot < 0) return;
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId + 1, static_cast<unsigned int>(t));
    return;
  }
  const uint32_t* v = reinterpret_cast<const uint32_t*>(
      a.v != nullptr ? static_cast<const __nv_bfloat16*>(a.v) + static_cast<long long>(t) * a.ldv
                     : k);
  uint32_t* kc = reinterpret_cast<uint32_t*>(a.kc) + slot * a.Hkv * dcp;
  uint32_t* vc = reinterpret_cast<uint32_t*>(a.vc) + slot * a.Hkv * dcp;
  for (int e = threadIdx.x; e < a.Hkv * dcp; e += blockDim.x) {
    const int h = e / dcp, c = e - h * dcp;
    kc[e] = c < dp ? turned(k, a.kw, ki, h * dp + c, c) : 0u;
    vc[e] = c < dp ? v[h * dp + c] : 0u;
  }
}

// The same for bf16 rows of whole 16-byte vectors (D, DC and rot multiples of 8): NV vectors per
// thread, queries then keys, read once and kept in registers.
template <int NV>
__global__ void __launch_bounds__(256) qk_norm_rope_cache_vec_kernel(const PrepArgs a) {
  __shared__ float red[2][8];
  const int t = blockIdx.x;
  const __nv_bfloat16* q =
      static_cast<const __nv_bfloat16*>(a.q) + static_cast<long long>(t) * a.ldq;
  const __nv_bfloat16* k =
      static_cast<const __nv_bfloat16*>(a.k) + static_cast<long long>(t) * a.ldk;
  const int dv = a.D / 8, dcv = a.DC / 8;
  const int vq = a.Hq * dv, vk = a.Hkv * dv;
  uint4 raw[NV];
  float sq = 0.0f, sk = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int e = threadIdx.x + i * 256;
    if (e >= vq + vk) continue;
    raw[i] = e < vq ? reinterpret_cast<const uint4*>(q)[e]
                    : reinterpret_cast<const uint4*>(k)[e - vq];
    const uint32_t w[4] = {raw[i].x, raw[i].y, raw[i].z, raw[i].w};
    float s = 0.0f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = unpack_bf16x2(w[j]);
      s += f.x * f.x + f.y * f.y;
    }
    if (e < vq) sq += s;
    else sk += s;
  }
  if (a.sumsq != nullptr) {
    sq = a.sumsq[2 * t];
    sk = a.sumsq[2 * t + 1];
  } else {
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) {
      red[0][threadIdx.x >> 5] = sq;
      red[1][threadIdx.x >> 5] = sk;
    }
    __syncthreads();
    sq = sk = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      sq += red[0][w];
      sk += red[1][w];
    }
  }
  const float qi = 1.0f / sqrtf(sq / static_cast<float>(a.q_all) + a.eps);
  const float ki = 1.0f / sqrtf(sk / static_cast<float>(a.k_all) + a.eps);
  long long pos = a.positions[t];
  if (pos < 0 || pos >= a.max_pos) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId, static_cast<unsigned int>(t));
    pos = 0;
  }
  long long slot = a.slots[t];
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId + 1, static_cast<unsigned int>(t));
    slot = -1;
  }
  const float* cs = a.cos_sin + pos * a.rot;
  uint4* qo = static_cast<uint4*>(a.qo) + static_cast<long long>(t) * a.Hq * dcv;
  uint4* kc = static_cast<uint4*>(a.kc) + slot * a.Hkv * dcv;
  uint4* vc = static_cast<uint4*>(a.vc) + slot * a.Hkv * dcv;
  const uint4* v = a.v != nullptr
      ? reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.v) +
                                       static_cast<long long>(t) * a.ldv) : nullptr;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int e = threadIdx.x + i * 256;
    if (e >= vq + vk) continue;
    const bool is_q = e < vq;
    const int x = is_q ? e : e - vq;
    if (!is_q && slot < 0) continue;
    const float inv = is_q ? qi : ki;
    const float4* w4 = reinterpret_cast<const float4*>(is_q ? a.qw : a.kw) + 2 * x;
    const float4 wa = w4[0], wb = w4[1];
    const float w[8] = {wa.x, wa.y, wa.z, wa.w, wb.x, wb.y, wb.z, wb.w};
    const uint32_t in[4] = {raw[i].x, raw[i].y, raw[i].z, raw[i].w};
    const int h = x / dv, c = x - h * dv;            // c: vector inside the head
    float co[4] = {1.0f, 1.0f, 1.0f, 1.0f}, si[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    if (c * 8 < a.rot) {
      const float4 cv = *reinterpret_cast<const float4*>(cs + c * 4);
      const float4 sv = *reinterpret_cast<const float4*>(cs + a.rot / 2 + c * 4);
      co[0] = cv.x; co[1] = cv.y; co[2] = cv.z; co[3] = cv.w;
      si[0] = sv.x; si[1] = sv.y; si[2] = sv.z; si[3] = sv.w;
    }
    uint32_t out[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = unpack_bf16x2(in[j]);
      const float u = f.x * inv * w[2 * j], y = f.y * inv * w[2 * j + 1];
      out[j] = pack_bf16x2(u * co[j] - y * si[j], y * co[j] + u * si[j]);
    }
    const uint4 res = make_uint4(out[0], out[1], out[2], out[3]);
    const int at = h * dcv + c;
    if (is_q) {
      qo[at] = res;
    } else {
      kc[at] = res;
      vc[at] = v != nullptr ? v[x] : raw[i];
    }
  }
  if (dcv == dv) return;
  const int pad = dcv - dv;
  for (int e = threadIdx.x; e < (a.Hq + a.Hkv) * pad; e += 256) {
    const int h = e / pad, c = dv + e - h * pad;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    if (h < a.Hq) {
      qo[h * dcv + c] = zero;
    } else if (slot >= 0) {
      kc[(h - a.Hq) * dcv + c] = zero;
      vc[(h - a.Hq) * dcv + c] = zero;
    }
  }
}

// ---------------------------------------------------------------------------
struct HeadNormArgs {
  const void* q;             // [T, Hq * D] view, row pitch ldq
  const void* k;             // [T, Hkv * D]
  const void* v;             // [T, Hkv * VD]
  const float* qw;           // [D]
  const float* kw;           // [D]
  const long long* slots;    // [T] (-1: no cache write)
  void* qo;                  // [T, Hq, DC]
  void* kc;                  // [num_slots, Hkv, DC]
  void* vc;
  long long ldq, ldk, ldv, num_slots;
  int T, Hq, Hkv, D, VD, DC;
  float eps;
  unsigned int* status;
};

template <typename T, int V>
__device__ __forceinline__ void load_elems(const T* p, float (&f)[V]) {
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
template <typename T, int V>
__device__ __forceinline__ void store_elems(T* p, const float (&f)[V]) {
  if constexpr (V == 4 && sizeof(T) == 2)
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  else if constexpr (V == 4)
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else
    p[0] = from_f32<T>(f[0]);
}

constexpr int kHeadWarps = 8;

// NI vectors of V elements per lane cover a head: 32 * V * NI >= DC
template <typename T, int V, int NI>
__global__ void __launch_bounds__(kHeadWarps * 32) head_norm_cache_kernel(const HeadNormArgs a) {
  const int lane = threadIdx.x & 31;
  const int per_token = a.Hq + 2 * a.Hkv;
  const long long job = static_cast<long long>(blockIdx.x) * kHeadWarps + (threadIdx.x >> 5);
  const int t = static_cast<int>(job / per_token);
  if (t >= a.T) return;
  const int j = static_cast<int>(job - static_cast<long long>(t) * per_token);
  const bool is_q = j < a.Hq, is_v = j >= a.Hq + a.Hkv;
  const int h = is_q ? j : (is_v ? j - a.Hq - a.Hkv : j - a.Hq);
  const int D = is_v ? a.VD : a.D;
  long long slot = 0;
  if (!is_q) {
    slot = a.slots[t];
    if (slot < 0) return;
    if (slot >= a.num_slots) {
      if (lane == 0)
        report_status(a.status, kStatusBounds, kKernelId + 1, static_cast<unsigned int>(t));
      return;
    }
  }
  const T* src = is_q ? static_cast<const T*>(a.q) + t * a.ldq + static_cast<long long>(h) * D
                      : (is_v ? static_cast<const T*>(a.v) + t * a.ldv + static_cast<long long>(h) * D
                              : static_cast<const T*>(a.k) + t * a.ldk + static_cast<long long>(h) * D);
  T* dst = is_q ? static_cast<T*>(a.qo) + (static_cast<long long>(t) * a.Hq + h) * a.DC
                : static_cast<T*>(is_v ? a.vc : a.kc) + (slot * a.Hkv + h) * a.DC;
  float x[NI][V];
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (i * 32 + lane) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) x[i][e] = 0.0f;
    if (c < D) load_elems<T, V>(src + c, x[i]);
#pragma unroll
    for (int e = 0; e < V; ++e) ss += x[i][e] * x[i][e];
  }
  if (!is_v) {
    const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(D) + a.eps);
    const float* w = is_q ? a.qw : a.kw;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = (i * 32 + lane) * V;
      if (c >= D) continue;
      float g[V];
      load_elems<float, V>(w + c, g);
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] *= inv * g[e];
    }
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (i * 32 + lane) * V;
    if (c < a.DC) store_elems<T, V>(dst + c, x[i]);
  }
}

template <typename T>
static int launch_head_norm(const HeadNormArgs& a, bool v4, cudaStream_t s) {
  const long long warps = static_cast<long long>(a.T) * (a.Hq + 2 * a.Hkv);
  const unsigned int grid = static_cast<unsigned int>((warps + kHeadWarps - 1) / kHeadWarps);
#define B200_HN(V, NI) head_norm_cache_kernel<T, V, NI><<<grid, kHeadWarps * 32, 0, s>>>(a)
  if (v4) {
    if (a.DC <= 128) B200_HN(4, 1);
    else if (a.DC <= 256) B200_HN(4, 2);
    else B200_HN(4, 4);
  } else {
    if (a.DC <= 128) B200_HN(1, 4);
    else B200_HN(1, 16);
  }
#undef B200_HN
  return static_cast<int>(cudaGetLastError());
}

// ---------------------------------------------------------------------------
struct QkvArgs {
  const void* q;             // [T, Hq * D] view, row pitch ldq
  const void* k;             // [T, Hkv * D]
  const void* v;             // [T, Hkv * VD]
  const float* qw;           // [Hq * D] norm weights, or null: no norm
  const float* kw;           // [Hkv * D]
  const float* sumsq;        // [T, 2] sums of squares of the whole q / k rows, or null: these rows
  const float* cos_sin;      // [positions, rot] cos | sin, or null with rot = 0
  const float* share;        // scalar: part of the first layer's values, or null: no mixing
  const void* first;         // [num_slots, first_pitch] value cache of that layer
  const long long* positions;
  const long long* slots;    // [T] (-1: no cache write)
  void* qo;                  // [T, Hq, DC]
  void* kc;                  // [num_slots, Hkv, DC]
  void* vc;
  long long ldq, ldk, ldv, num_slots, max_pos, first_pitch;
  int T, Hq, Hkv, D, VD, DC, rot, q_all, k_all, v_norm;
  int first_dim, first_dc;   // value and cached width of a head in the first layer's cache
  int temp_every;
  float temp, eps;           // temp 0: none
  unsigned int* status;
};

constexpr int kMaxKvHeads = 256;

// Position (clamped, a bad one is reported), cache slot (-1: none) and query factor of a token.
struct TokenRow {
  long long pos, slot;
  float factor;
};
__device__ __forceinline__ TokenRow token_row(const QkvArgs& a, int t) {
  TokenRow r{a.positions[t], a.slots[t], 1.0f};
  if (a.rot > 0 && (r.pos < 0 || r.pos >= a.max_pos)) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId + 4, static_cast<unsigned int>(t));
    r.pos = 0;
  }
  if (r.slot >= a.num_slots) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId + 5, static_cast<unsigned int>(t));
    r.slot = -1;
  }
  if (a.temp != 0.0f)
    r.factor = 1.0f + a.temp * logf(static_cast<float>((r.pos + 1) / a.temp_every) + 1.0f);
  return r;
}

template <typename T>
__global__ void __launch_bounds__(256) qkv_cache_kernel(const QkvArgs a) {
  __shared__ float red[32];
  __shared__ float s_vinv[kMaxKvHeads];
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  const T* q = static_cast<const T*>(a.q) + static_cast<long long>(t) * a.ldq;
  const T* k = static_cast<const T*>(a.k) + static_cast<long long>(t) * a.ldk;
  const T* v = static_cast<const T*>(a.v) + static_cast<long long>(t) * a.ldv;
  float qi = 1.0f, ki = 1.0f;
  if (a.qw != nullptr) {
    float sq = 0.0f, sk = 0.0f;
    if (a.sumsq != nullptr) {
      sq = a.sumsq[2 * t];
      sk = a.sumsq[2 * t + 1];
    } else {
      for (int c = threadIdx.x; c < a.Hq * a.D; c += blockDim.x) {
        const float f = to_f32<T>(q[c]);
        sq += f * f;
      }
      for (int c = threadIdx.x; c < a.Hkv * a.D; c += blockDim.x) {
        const float f = to_f32<T>(k[c]);
        sk += f * f;
      }
      sq = block_sum(sq, red);
      sk = block_sum(sk, red);
    }
    qi = 1.0f / sqrtf(sq / static_cast<float>(a.q_all) + a.eps);
    ki = 1.0f / sqrtf(sk / static_cast<float>(a.k_all) + a.eps);
  }
  for (int h = threadIdx.x >> 5; h < a.Hkv; h += blockDim.x >> 5) {
    float inv = 1.0f;
    if (a.v_norm) {
      float ss = 0.0f;
      for (int c = lane; c < a.VD; c += 32) {
        const float f = to_f32<T>(v[h * a.VD + c]);
        ss += f * f;
      }
      inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(a.VD) + a.eps);
    }
    if (lane == 0) s_vinv[h] = inv;
  }
  __syncthreads();
  const TokenRow row = token_row(a, t);
  const float* cs = a.rot > 0 ? a.cos_sin + row.pos * a.rot : nullptr;
  const int half = a.rot / 2;
  auto turned = [&](const T* x, const float* w, float inv, int base, int c) {
    auto at = [&](int i) {
      const float f = to_f32<T>(x[base + i]) * inv;
      return w != nullptr ? f * w[base + i] : f;
    };
    const float self = at(c);
    if (c >= a.rot) return self;
    const bool lower = c < half;
    const int i = lower ? c : c - half;
    const float other = at(lower ? c + half : c - half);
    return lower ? self * cs[i] - other * cs[half + i] : self * cs[i] + other * cs[half + i];
  };
  T* qo = static_cast<T*>(a.qo) + static_cast<long long>(t) * a.Hq * a.DC;
  for (int e = threadIdx.x; e < a.Hq * a.DC; e += blockDim.x) {
    const int h = e / a.DC, c = e - h * a.DC;
    qo[e] = from_f32<T>(c < a.D ? turned(q, a.qw, qi, h * a.D, c) * row.factor : 0.0f);
  }
  if (row.slot < 0) return;
  T* kc = static_cast<T*>(a.kc) + row.slot * a.Hkv * a.DC;
  T* vc = static_cast<T*>(a.vc) + row.slot * a.Hkv * a.DC;
  const T* first = a.share != nullptr ? static_cast<const T*>(a.first) + row.slot * a.first_pitch
                                      : nullptr;
  const float share = a.share != nullptr ? *a.share : 0.0f;
  for (int e = threadIdx.x; e < a.Hkv * a.DC; e += blockDim.x) {
    const int h = e / a.DC, c = e - h * a.DC;
    kc[e] = from_f32<T>(c < a.D ? turned(k, a.kw, ki, h * a.D, c) : 0.0f);
    float f = 0.0f;
    if (c < a.VD) {
      const int i = h * a.VD + c;
      f = to_f32<T>(v[i]) * s_vinv[h];
      if (first != nullptr) {
        const int fh = i / a.first_dim;
        f = (1.0f - share) * f +
            share * to_f32<T>(first[fh * a.first_dc + i - fh * a.first_dim]);
      }
    }
    vc[e] = from_f32<T>(f);
  }
}

__device__ __forceinline__ void unpack8(const uint4& u, float (&f)[8]) {
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 p = unpack_bf16x2(w[j]);
    f[2 * j] = p.x;
    f[2 * j + 1] = p.y;
  }
}
__device__ __forceinline__ uint4 pack8(const float (&f)[8]) {
  return make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]),
                    pack_bf16x2(f[6], f[7]));
}
__device__ __forceinline__ void load8f(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  const float4 b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

// The same for bf16 rows of whole 16-byte vectors.  A thread holds NV pairs of vectors, queries
// then keys: the two that turn with each other, or two neighbours behind the rotated dimensions
// (D and rot multiples of 16, VD and DC of 8, VD <= 256).
template <int NV>
__global__ void __launch_bounds__(256) qkv_cache_vec_kernel(const QkvArgs a) {
  __shared__ float red[2][8];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const __nv_bfloat16* q =
      static_cast<const __nv_bfloat16*>(a.q) + static_cast<long long>(t) * a.ldq;
  const __nv_bfloat16* k =
      static_cast<const __nv_bfloat16*>(a.k) + static_cast<long long>(t) * a.ldk;
  const int per = a.D / 16, nq = a.Hq * per, nk = a.Hkv * per, turned = a.rot / 16;
  uint4 raw[NV][2];
  int at[NV], step[NV];                          // first element of the pair, distance to its mate
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int e = threadIdx.x + i * 256;
    if (e >= nq + nk) continue;
    const int x = e < nq ? e : e - nq;
    const int h = x / per, c = x - h * per;
    at[i] = h * a.D + (c < turned ? c * 8 : a.rot + (c - turned) * 16);
    step[i] = c < turned ? a.rot / 2 : 8;
    const __nv_bfloat16* src = (e < nq ? q : k) + at[i];
    raw[i][0] = *reinterpret_cast<const uint4*>(src);
    raw[i][1] = *reinterpret_cast<const uint4*>(src + step[i]);
  }
  const TokenRow row = token_row(a, t);
  // values: one warp per head
  if (row.slot >= 0) {
    const int vv = a.VD / 8, cv = a.DC / 8;
    const uint4* v = reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.v) +
                                                    static_cast<long long>(t) * a.ldv);
    uint4* vc = static_cast<uint4*>(a.vc) + row.slot * a.Hkv * cv;
    const float share = a.share != nullptr ? *a.share : 0.0f;
    for (int h = warp; h < a.Hkv; h += 8) {
      float f[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f}, g[8];
      if (lane < vv) {
        unpack8(v[h * vv + lane], f);
        if (a.share != nullptr) {
          const int e = h * a.VD + lane * 8, fh = e / a.first_dim;
          unpack8(*reinterpret_cast<const uint4*>(
                      static_cast<const __nv_bfloat16*>(a.first) + row.slot * a.first_pitch +
                      fh * a.first_dc + e - fh * a.first_dim), g);
        }
      }
      if (a.v_norm) {
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
        const float inv = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(a.VD) + a.eps);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= inv;
      }
      if (a.share != nullptr && lane < vv) {
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = (1.0f - share) * f[j] + share * g[j];
      }
      for (int c = lane; c < cv; c += 32)        // zeros behind the value's columns
        vc[h * cv + c] = c < vv ? pack8(f) : make_uint4(0, 0, 0, 0);
    }
  }
  float qi = row.factor, ki = 1.0f;
  if (a.qw != nullptr) {
    float sq = 0.0f, sk = 0.0f;
    if (a.sumsq != nullptr) {
      sq = a.sumsq[2 * t];
      sk = a.sumsq[2 * t + 1];
    } else {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int e = threadIdx.x + i * 256;
        if (e >= nq + nk) continue;
        float s = 0.0f;
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          float f[8];
          unpack8(raw[i][m], f);
#pragma unroll
          for (int j = 0; j < 8; ++j) s += f[j] * f[j];
        }
        if (e < nq) sq += s;
        else sk += s;
      }
      sq = warp_sum(sq);
      sk = warp_sum(sk);
      if (lane == 0) {
        red[0][warp] = sq;
        red[1][warp] = sk;
      }
      __syncthreads();
      sq = sk = 0.0f;
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        sq += red[0][w];
        sk += red[1][w];
      }
    }
    qi = row.factor / sqrtf(sq / static_cast<float>(a.q_all) + a.eps);
    ki = 1.0f / sqrtf(sk / static_cast<float>(a.k_all) + a.eps);
  }
  const float* cs = a.rot > 0 ? a.cos_sin + row.pos * a.rot : nullptr;
  __nv_bfloat16* qo =
      static_cast<__nv_bfloat16*>(a.qo) + static_cast<long long>(t) * a.Hq * a.DC;
  __nv_bfloat16* kc = static_cast<__nv_bfloat16*>(a.kc) + row.slot * a.Hkv * a.DC;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int e = threadIdx.x + i * 256;
    if (e >= nq + nk) continue;
    const bool is_q = e < nq;
    if (!is_q && row.slot < 0) continue;
    const float inv = is_q ? qi : ki;
    float f[2][8];
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      unpack8(raw[i][m], f[m]);
      if (a.qw != nullptr) {
        float w[8];
        load8f((is_q ? a.qw : a.kw) + at[i] + m * step[i], w);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[m][j] *= inv * w[j];
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) f[m][j] *= inv;
      }
    }
    const int h = at[i] / a.D, c = at[i] - h * a.D;
    if (c < a.rot) {
      float co[8], si[8];
      load8f(cs + c, co);
      load8f(cs + a.rot / 2 + c, si);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float u = f[0][j], w = f[1][j];
        f[0][j] = u * co[j] - w * si[j];
        f[1][j] = w * co[j] + u * si[j];
      }
    }
    __nv_bfloat16* dst = (is_q ? qo : kc) + h * a.DC + c;
    *reinterpret_cast<uint4*>(dst) = pack8(f[0]);
    *reinterpret_cast<uint4*>(dst + step[i]) = pack8(f[1]);
  }
  if (a.DC == a.D) return;
  const int pad = (a.DC - a.D) / 8;
  for (int e = threadIdx.x; e < (a.Hq + a.Hkv) * pad; e += 256) {
    const int h = e / pad, c = a.D + (e - h * pad) * 8;
    if (h >= a.Hq && row.slot < 0) continue;
    __nv_bfloat16* dst = h < a.Hq ? qo + h * a.DC + c : kc + (h - a.Hq) * a.DC + c;
    *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
  }
}

// ---------------------------------------------------------------------------
struct AttnArgs {
  const void* q;             // [T, Hq, DC]
  const void* kc;            // [num_slots, Hkv, DC]
  const void* vc;
  void* out;                 // [T, Hq, OD], row pitch ldo: the first OD of the DC columns
  const int* block_tables;   // [B, max_blocks]
  const int* seq_lens;       // [B]
  const int* cu_q;           // [num_prefills + 1] relative to token num_decodes, or null
  const float* sink;         // [Hq] or null
  long long num_slots, ldo;
  int T, Hq, Hkv, DC, OD, num_decodes, num_prefills, max_blocks, block_size;
  int chunk;                 // > 0: keys of the query's own chunk of that many positions
  int window;                // > 0: the last keys up to the query
  const float* slopes;       // [Hq] distance biases: slope * (query - key position) comes off, or null
  float scale, softcap;      // softcap > 0: scores become softcap * tanh(score / softcap)
  unsigned int* status;
};

constexpr int kWarps = 4;      // warps that share the keys of one (token, head)
constexpr int kBatch = 4;      // keys a warp has in flight

template <typename T, int NC>
__global__ void __launch_bounds__(kWarps * 32) any_attention_kernel(const AttnArgs a) {
  __shared__ float s_m[kWarps], s_l[kWarps];
  __shared__ float s_o[kWarps][NC * 32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x, head = blockIdx.y;
  const int kvh = head / (a.Hq / a.Hkv);
  const TokenPlace pl = token_place(t, a.num_decodes, a.num_prefills, a.cu_q);
  int keys = 0;
  if (pl.req >= 0) {
    keys = a.seq_lens[pl.req];
    if (t >= a.num_decodes)      // tokens of the request behind this one in the step
      keys -= a.cu_q[pl.req - a.num_decodes + 1] - (t - a.num_decodes) - 1;
  }
  if (keys > a.max_blocks * a.block_size) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId + 2, static_cast<unsigned int>(t));
    keys = 0;
  }
  const long long row = (static_cast<long long>(t) * a.Hq + head) * a.DC;
  float q[NC], acc[NC];
#pragma unroll
  for (int i = 0; i < NC; ++i) {
    const int c = lane + 32 * i;
    q[i] = c < a.DC ? to_f32<T>(static_cast<const T*>(a.q)[row + c]) : 0.0f;
    acc[i] = 0.0f;
  }
  float m = -INFINITY, l = 0.0f;
  const int* bt = a.block_tables + static_cast<long long>(pl.req < 0 ? 0 : pl.req) * a.max_blocks;
  int first = a.chunk > 0 && keys > 0 ? (keys - 1) / a.chunk * a.chunk : 0;
  if (a.window > 0) first = max(first, keys - a.window);
  const float slope = a.slopes != nullptr ? a.slopes[head] : 0.0f;
  for (int k0 = first + warp * kBatch; k0 < keys; k0 += kWarps * kBatch) {
    float s[kBatch], v[kBatch][NC];
#pragma unroll
    for (int b = 0; b < kBatch; ++b) {
      const int key = k0 + b;
      long long slot = -1;
      if (key < keys) {
        slot = static_cast<long long>(bt[key / a.block_size]) * a.block_size + key % a.block_size;
        if (slot < 0 || slot >= a.num_slots) {
          if (lane == 0)
            report_status(a.status, kStatusBounds, kKernelId + 3, static_cast<unsigned int>(t));
          slot = -1;
        }
      }
      const long long at = (slot * a.Hkv + kvh) * a.DC;
      float d = 0.0f;
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int c = lane + 32 * i;
        const bool in = slot >= 0 && c < a.DC;
        d += in ? q[i] * to_f32<T>(static_cast<const T*>(a.kc)[at + c]) : 0.0f;
        v[b][i] = in ? to_f32<T>(static_cast<const T*>(a.vc)[at + c]) : 0.0f;
      }
      s[b] = d;
    }
    float top = m;
#pragma unroll
    for (int b = 0; b < kBatch; ++b) {
      s[b] = k0 + b < keys ? warp_sum(s[b]) * a.scale : -INFINITY;
      if (a.softcap > 0.0f && k0 + b < keys) s[b] = a.softcap * tanhf(s[b] / a.softcap);
      if (a.slopes != nullptr && k0 + b < keys)
        s[b] -= slope * static_cast<float>(keys - 1 - k0 - b);
      top = fmaxf(top, s[b]);
    }
    const float al = expf(m - top);            // top is finite: key k0 is visible
    m = top;
    l *= al;
#pragma unroll
    for (int i = 0; i < NC; ++i) acc[i] *= al;
#pragma unroll
    for (int b = 0; b < kBatch; ++b) {
      const float p = expf(s[b] - m);
      l += p;
#pragma unroll
      for (int i = 0; i < NC; ++i) acc[i] += p * v[b][i];
    }
  }
  if (lane == 0) {
    s_m[warp] = m;
    s_l[warp] = l;
  }
#pragma unroll
  for (int i = 0; i < NC; ++i) s_o[warp][lane + 32 * i] = acc[i];
  __syncthreads();
  float top = a.sink != nullptr ? a.sink[head] : -INFINITY;
  const float sink = top;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) top = fmaxf(top, s_m[w]);
  float f[kWarps], den = a.sink != nullptr ? expf(sink - top) : 0.0f;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) {
    f[w] = s_m[w] == -INFINITY ? 0.0f : expf(s_m[w] - top);
    den += s_l[w] * f[w];
  }
  const float inv = keys > 0 ? 1.0f / den : 0.0f;
  T* out = static_cast<T*>(a.out) + static_cast<long long>(t) * a.ldo +
           static_cast<long long>(head) * a.OD;
  for (int c = threadIdx.x; c < a.OD; c += blockDim.x) {
    float o = 0.0f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) o += s_o[w][c] * f[w];
    out[c] = from_f32<T>(o * inv);
  }
}

template <typename T>
static int dispatch_attention(const AttnArgs& a, cudaStream_t s) {
  const int nc = (a.DC + 31) / 32;
  dim3 grid(a.T, a.Hq);
  if (nc <= 2) any_attention_kernel<T, 2><<<grid, kWarps * 32, 0, s>>>(a);
  else if (nc <= 4) any_attention_kernel<T, 4><<<grid, kWarps * 32, 0, s>>>(a);
  else if (nc <= 8) any_attention_kernel<T, 8><<<grid, kWarps * 32, 0, s>>>(a);
  else if (nc <= 16) any_attention_kernel<T, 16><<<grid, kWarps * 32, 0, s>>>(a);
  else return -20;
  return static_cast<int>(cudaGetLastError());
}

}  // namespace anyattn
}  // namespace b200

using namespace b200;
using namespace b200::anyattn;

// dtype (rows and caches): 0 bf16, 2 fp32.  rot even, <= D.  q_all / k_all: number of elements a
// norm runs over (with sumsq, rows of other ranks included).
B200_API int b200_qk_norm_rope_cache(const void* q, long long ldq, const void* k, long long ldk,
                                     const void* v, long long ldv, const float* qw, const float* kw,
                                     const float* sumsq, int q_all, int k_all, float eps,
                                     const float* cos_sin, int rot, long long max_pos, int is_neox,
                                     const long long* positions, const long long* slots, void* qo,
                                     void* kc, void* vc, long long num_slots, int T, int Hq,
                                     int Hkv, int D, int DC, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (Hq <= 0 || Hkv <= 0 || D <= 0 || DC < D || rot < 0 || rot > D || (rot & 1) != 0 ||
      (dtype != 0 && dtype != 2))
    return -2;
  PrepArgs a;
  a.q = q; a.k = k; a.v = v; a.qw = qw; a.kw = kw; a.sumsq = sumsq; a.cos_sin = cos_sin;
  a.positions = positions; a.slots = slots; a.qo = qo; a.kc = kc; a.vc = vc; a.ldq = ldq;
  a.ldk = ldk; a.ldv = ldv; a.num_slots = num_slots; a.max_pos = max_pos; a.T = T; a.Hq = Hq;
  a.Hkv = Hkv; a.D = D; a.DC = DC; a.rot = rot; a.q_all = q_all; a.k_all = k_all;
  a.is_neox = is_neox; a.eps = eps; a.status = status_ptr();
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const auto even = [](const void* p, int bytes) {
    return (reinterpret_cast<uintptr_t>(p) % bytes) == 0;
  };
  const int vectors = (Hq + Hkv) * D / 8;
  const bool vec = dtype == 0 && !is_neox && (D % 8) == 0 && (DC % 8) == 0 && (rot % 8) == 0 &&
                   (ldq % 8) == 0 && (ldk % 8) == 0 && (ldv % 8) == 0 && even(q, 16) &&
                   even(k, 16) && even(v, 16) && even(qw, 16) && even(kw, 16) &&
                   even(cos_sin, 16) && even(qo, 16) && even(kc, 16) && even(vc, 16) &&
                   vectors <= 8 * 256;
  if (vec) {
    if (vectors <= 256) qk_norm_rope_cache_vec_kernel<1><<<T, 256, 0, s>>>(a);
    else if (vectors <= 512) qk_norm_rope_cache_vec_kernel<2><<<T, 256, 0, s>>>(a);
    else if (vectors <= 1024) qk_norm_rope_cache_vec_kernel<4><<<T, 256, 0, s>>>(a);
    else qk_norm_rope_cache_vec_kernel<8><<<T, 256, 0, s>>>(a);
  } else if (dtype == 2)
    qk_norm_rope_cache_kernel<float><<<T, 256, 0, s>>>(a);
  else if (!is_neox && (D & 1) == 0 && (DC & 1) == 0 && (ldq & 1) == 0 && (ldk & 1) == 0 &&
           (ldv & 1) == 0 && even(q, 4) && even(k, 4) && even(v, 4) && even(qw, 8) &&
           even(kw, 8) && even(qo, 4) && even(kc, 4) && even(vc, 4))
    qk_norm_rope_cache_pairs_kernel<<<T, 256, 0, s>>>(a);
  else
    qk_norm_rope_cache_kernel<__nv_bfloat16><<<T, 256, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

// dtype (rows and caches): 0 bf16, 2 fp32.  q [T, Hq * D], k [T, Hkv * D], v [T, Hkv * VD] views;
// D, VD <= DC <= 512.
B200_API int b200_head_norm_cache(const void* q, long long ldq, const void* k, long long ldk,
                                  const void* v, long long ldv, const float* qw, const float* kw,
                                  float eps, const long long* slots, void* qo, void* kc, void* vc,
                                  long long num_slots, int T, int Hq, int Hkv, int D, int VD, int DC,
                                  int dtype, void* stream) {
  if (T <= 0) return 0;
  if (Hq <= 0 || Hkv <= 0 || D <= 0 || VD <= 0 || DC < D || DC < VD || DC > 512 ||
      (dtype != 0 && dtype != 2))
    return -2;
  HeadNormArgs a;
  a.q = q; a.k = k; a.v = v; a.qw = qw; a.kw = kw; a.slots = slots; a.qo = qo; a.kc = kc;
  a.vc = vc; a.ldq = ldq; a.ldk = ldk; a.ldv = ldv; a.num_slots = num_slots; a.T = T; a.Hq = Hq;
  a.Hkv = Hkv; a.D = D; a.VD = VD; a.DC = DC; a.eps = eps; a.status = status_ptr();
  const auto at = [](const void* p, int bytes) {
    return (reinterpret_cast<uintptr_t>(p) % bytes) == 0;
  };
  const int vb = dtype == 0 ? 8 : 16;
  const bool v4 = (D % 4) == 0 && (VD % 4) == 0 && (DC % 4) == 0 && (ldq % 4) == 0 &&
                  (ldk % 4) == 0 && (ldv % 4) == 0 && at(q, vb) && at(k, vb) && at(v, vb) &&
                  at(qo, vb) && at(kc, vb) && at(vc, vb) && at(qw, 16) && at(kw, 16);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == 0 ? launch_head_norm<__nv_bfloat16>(a, v4, s) : launch_head_norm<float>(a, v4, s);
}

// dtype (rows and caches): 0 bf16, 2 fp32.  q [T, Hq * D], k [T, Hkv * D], v [T, Hkv * VD] views; D,
// VD <= DC <= 512.  qw / kw null: no norm.  temp: queries times 1 + temp * ln(floor((p + 1) /
// temp_every) + 1).  share / first: values become (1 - share) * own + share * first, `first` a value
// cache [num_slots, heads, first_dc] whose first first_dim columns of a head are in use, read at the
// token's own slot.
B200_API int b200_qkv_cache(const void* q, long long ldq, const void* k, long long ldk,
                            const void* v, long long ldv, const float* qw, const float* kw,
                            const float* sumsq, int q_all, int k_all, float eps,
                            const float* cos_sin, int rot, long long max_pos, float temp,
                            int temp_every, int v_norm, const float* share, const void* first,
                            long long first_pitch, int first_dim, int first_dc,
                            const long long* positions, const long long* slots, void* qo, void* kc,
                            void* vc, long long num_slots, int T, int Hq, int Hkv, int D, int VD,
                            int DC, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (Hq <= 0 || Hkv <= 0 || D <= 0 || VD <= 0 || DC < D || DC < VD || rot < 0 || rot > D ||
      (rot & 1) != 0 || (rot > 0 && cos_sin == nullptr) || (qw == nullptr) != (kw == nullptr) ||
      temp_every < 1 || (share != nullptr && (first == nullptr || first_dim <= 0)) ||
      (dtype != 0 && dtype != 2))
    return -2;
  if (Hkv > kMaxKvHeads) return -20;
  QkvArgs a;
  a.q = q; a.k = k; a.v = v; a.qw = qw; a.kw = kw; a.sumsq = sumsq; a.cos_sin = cos_sin;
  a.share = share; a.first = first; a.positions = positions; a.slots = slots; a.qo = qo; a.kc = kc;
  a.vc = vc; a.ldq = ldq; a.ldk = ldk; a.ldv = ldv; a.num_slots = num_slots; a.max_pos = max_pos;
  a.first_pitch = first_pitch; a.T = T; a.Hq = Hq; a.Hkv = Hkv; a.D = D; a.VD = VD; a.DC = DC;
  a.rot = rot; a.q_all = q_all; a.k_all = k_all; a.v_norm = v_norm; a.first_dim = first_dim;
  a.first_dc = first_dc; a.temp_every = temp_every; a.temp = temp; a.eps = eps;
  a.status = status_ptr();
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const auto at = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const int pairs = (Hq + Hkv) * D / 16;
  const bool vec = dtype == 0 && (D % 16) == 0 && (rot % 16) == 0 && (VD % 8) == 0 && VD <= 256 &&
                   (DC % 8) == 0 && (ldq % 8) == 0 && (ldk % 8) == 0 && (ldv % 8) == 0 &&
                   (share == nullptr || ((first_dim % 8) == 0 && (first_dc % 8) == 0 &&
                                         (first_pitch % 8) == 0)) &&
                   at(q) && at(k) && at(v) && at(qw) && at(kw) && at(cos_sin) && at(first) &&
                   at(qo) && at(kc) && at(vc) && pairs <= 8 * 256;
  if (vec) {
    if (pairs <= 256) qkv_cache_vec_kernel<1><<<T, 256, 0, s>>>(a);
    else if (pairs <= 512) qkv_cache_vec_kernel<2><<<T, 256, 0, s>>>(a);
    else if (pairs <= 1024) qkv_cache_vec_kernel<4><<<T, 256, 0, s>>>(a);
    else qkv_cache_vec_kernel<8><<<T, 256, 0, s>>>(a);
  } else if (dtype == 2) {
    qkv_cache_kernel<float><<<T, 256, 0, s>>>(a);
  } else {
    qkv_cache_kernel<__nv_bfloat16><<<T, 256, 0, s>>>(a);
  }
  return static_cast<int>(cudaGetLastError());
}

// q [T, Hq, DC], out [T, Hq, OD] with row pitch ldo (the first OD <= DC columns of a head's value);
// softcap / chunk / window 0 and slopes null: none.  -20: a head dimension the kernel does not cover (> 512).
B200_API int b200_any_attention(const void* q, const void* kc, const void* vc, long long num_slots,
                                void* out, long long ldo, int OD, const int* block_tables,
                                int max_blocks, int block_size, const int* seq_lens,
                                const int* cu_q, const float* sink, int T, int Hq, int Hkv, int DC,
                                int num_decodes, int num_prefills, float scale, float softcap,
                                int chunk, int window, const float* slopes, int dtype,
                                void* stream) {
  if (T <= 0) return 0;
  if (window < 0 || Hq <= 0 || Hkv <= 0 || Hq % Hkv != 0 || DC <= 0 || OD <= 0 || OD > DC || block_size <= 0 ||
      Hq > 65535 || chunk < 0 || (dtype != 0 && dtype != 2))
    return -2;
  AttnArgs a;
  a.q = q; a.kc = kc; a.vc = vc; a.out = out; a.block_tables = block_tables;
  a.seq_lens = seq_lens; a.cu_q = cu_q; a.sink = sink; a.num_slots = num_slots; a.T = T; a.Hq = Hq;
  a.Hkv = Hkv; a.DC = DC; a.num_decodes = num_decodes; a.num_prefills = num_prefills;
  a.max_blocks = max_blocks; a.block_size = block_size; a.scale = scale; a.status = status_ptr();
  a.ldo = ldo; a.OD = OD; a.softcap = softcap; a.chunk = chunk;
  a.window = window; a.slopes = slopes;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == 0 ? dispatch_attention<__nv_bfloat16>(a, s) : dispatch_attention<float>(a, s);
}
