// Latent attention: cache update and the general attention kernel.
//
//   latent_cache     RMSNorm of the latent projection -> one padded row per token in the paged
//                    latent cache; in the same pass the last row of a token-shifted input that a
//                    portion (or a cache block) holds goes to the block's state row.  With a
//                    rotated part, R columns behind the latent: those of the key are rotated into
//                    the cache row, those of every query head into its latent query
//   latent_attention any head count and latent width, fp32 or bf16 rows: one warp per
//                    (token, head), key tiles staged in shared memory as fp32, online softmax.
//                    The tcgen05 kernel (attention_mla.cu) takes the layouts it covers; this one
//                    serves models that run in 32-bit and the remaining shapes.
//
// The value of a key is its own cached row, so the output is in latent space; what it holds behind
// the latent columns meets zero rows of the matrix that expands it.
#include "common.cuh"

namespace b200 {
namespace latent {

constexpr unsigned int kKernelId = 70;

struct CacheArgs {
  const void* kv;            // [T, ldkv] latent projection (view of a wider row), L + R columns
  const void* weight;        // [L]
  void* cache;               // [num_slots, W]
  const long long* slots;    // [T] (-1: no write)
  const float* x;            // [T, H] rows whose last one per block is kept, or null
  float* state;              // [num_blocks, H]
  const int* cu_q;
  const void* q;             // [T, ldq] view: per head dim + R columns, the last R rotated
  void* q_lat;               // [T, N, W] latent queries: columns L .. L + R are written
  const float* cos_sin;      // [max_pos, R] cos | sin
  const long long* positions;
  long long ldkv, num_slots, ldq, max_pos;
  int T, L, W, H, R, N, dim, num_decodes, num_prefills, block_size;
  float eps;
  unsigned int* status;
};

// (u, v) at positions 2 i, 2 i + 1 turned by the angle of (co, si)
template <typename T, bool kPairs>
__device__ __forceinline__ void rotate_pair(const T* src, T* dst, float co, float si) {
  float u, v;
  if constexpr (kPairs && sizeof(T) == 2) {
    const float2 f = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(src));
    u = f.x; v = f.y;
  } else {
    u = to_f32<T>(src[0]);
    v = to_f32<T>(src[1]);
  }
  const float a = u * co - v * si, b = v * co + u * si;
  if constexpr (kPairs && sizeof(T) == 2) {
    *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(a, b);
  } else {
    dst[0] = from_f32<T>(a);
    dst[1] = from_f32<T>(b);
  }
}

// kPairs: pairs of 16-bit elements are 4-byte aligned everywhere
template <typename T, bool kPairs>
__global__ void __launch_bounds__(128) latent_cache_kernel(const CacheArgs a) {
  __shared__ float red[32];
  const int t = blockIdx.x;
  const int half = a.R / 2;
  const float* cs = nullptr;
  if (a.R > 0) {
    long long pos = a.positions[t];
    if (pos < 0 || pos >= a.max_pos) {
      if (threadIdx.x == 0)
        report_status(a.status, kStatusBounds, kKernelId + 3, static_cast<unsigned int>(t));
      pos = 0;
    }
    cs = a.cos_sin + pos * a.R;
    const T* q = static_cast<const T*>(a.q) + static_cast<long long>(t) * a.ldq + a.dim;
    T* ql = static_cast<T*>(a.q_lat) + static_cast<long long>(t) * a.N * a.W + a.L;
    for (int e = threadIdx.x; e < a.N * half; e += blockDim.x) {
      const int h = e / half, i = e - h * half;
      rotate_pair<T, kPairs>(q + static_cast<long long>(h) * (a.dim + a.R) + 2 * i,
                             ql + static_cast<long long>(h) * a.W + 2 * i, cs[i], cs[half + i]);
    }
  }
  const long long slot = a.slots[t];
  if (slot < 0) return;
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId, static_cast<unsigned int>(t));
    return;
  }
  const T* kv = static_cast<const T*>(a.kv) + static_cast<long long>(t) * a.ldkv;
  // the state row first: its loads and stores overlap the latency of the norm
  if (a.x != nullptr) {
    const TokenPlace pl = token_place(t, a.num_decodes, a.num_prefills, a.cu_q);
    if (pl.last || (slot + 1) % a.block_size == 0) {
      const float* x = a.x + static_cast<long long>(t) * a.H;
      float* st = a.state + slot / a.block_size * a.H;
      if ((a.H % 4) == 0) {
#pragma unroll 4
        for (int c = threadIdx.x; c < a.H / 4; c += blockDim.x)
          reinterpret_cast<float4*>(st)[c] = reinterpret_cast<const float4*>(x)[c];
      } else {
        for (int c = threadIdx.x; c < a.H; c += blockDim.x) st[c] = x[c];
      }
    }
  }
  const T* w = static_cast<const T*>(a.weight);
  T* dst = static_cast<T*>(a.cache) + slot * a.W;
  constexpr int kKeep = 8;                 // columns per thread that stay in registers
  float v[kKeep];
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    v[i] = c < a.L ? to_f32<T>(kv[c]) : 0.0f;
    ss += v[i] * v[i];
  }
  for (int c = threadIdx.x + kKeep * blockDim.x; c < a.L; c += blockDim.x) {
    const float u = to_f32<T>(kv[c]);
    ss += u * u;
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / static_cast<float>(a.L) + a.eps);
  for (int i = threadIdx.x; i < half; i += blockDim.x)
    rotate_pair<T, kPairs>(kv + a.L + 2 * i, dst + a.L + 2 * i, cs[i], cs[half + i]);
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    if (c >= a.L && c < a.L + a.R) continue;
    if (c < a.W) dst[c] = from_f32<T>(c < a.L ? v[i] * inv * to_f32<T>(w[c]) : 0.0f);
  }
  for (int c = threadIdx.x + kKeep * blockDim.x; c < a.W; c += blockDim.x)
    if (c < a.L || c >= a.L + a.R) dst[c] = from_f32<T>(c < a.L ? to_f32<T>(kv[c]) * inv * to_f32<T>(w[c]) : 0.0f);
}

// ---------------------------------------------------------------------------
constexpr int kWarps = 8;      // heads per CTA
constexpr int kKeys = 32;      // keys per tile, one per lane

struct AttnArgs {
  const void* q;             // [T, N, W]
  const void* cache;         // [num_slots, W]
  void* out;                 // [T, N, W]
  const int* block_tables;   // [B, max_blocks]
  const int* seq_lens;       // [B]
  const int* cu_q;           // [num_prefills + 1] relative to token num_decodes, or null
  const float* sink;         // [N]: exp(sink) joins the denominator, or null
  const void* gate;          // [T, ldg]: head h's output times sigmoid(gate[t, h]), or null
  long long num_slots, ldg;
  int T, N, W, num_decodes, num_prefills, max_blocks, block_size;
  float scale;
  unsigned int* status;
};

// W floats per key row, padded so that float4 reads of 32 consecutive rows spread over the banks
__host__ __device__ constexpr int key_pitch(int W) { return W + 4; }

template <typename T, int NC>
__global__ void __launch_bounds__(kWarps * 32) latent_attention_kernel(const AttnArgs a) {
  extern __shared__ float4 smem4[];
  float* ks = reinterpret_cast<float*>(smem4);                 // [kKeys][pitch]
  const int pitch = key_pitch(a.W);
  float* qs = ks + kKeys * pitch;                              // [kWarps][W]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int head = blockIdx.y * kWarps + warp;
  const bool live = head < a.N;
  const long long orow = (static_cast<long long>(t) * a.N + head) * a.W;
  T* out = static_cast<T*>(a.out);
  const TokenPlace pl = token_place(t, a.num_decodes, a.num_prefills, a.cu_q);
  int keys = 0;
  if (pl.req >= 0) {
    const int n = a.seq_lens[pl.req];
    if (t < a.num_decodes) {
      keys = n;
    } else {
      // tokens of the request behind this one in the step
      const int behind = a.cu_q[pl.req - a.num_decodes + 1] - (t - a.num_decodes) - 1;
      keys = n - behind;
    }
  }
  if (keys > a.max_blocks * a.block_size) {
    if (threadIdx.x == 0)
      report_status(a.status, kStatusBounds, kKernelId + 1, static_cast<unsigned int>(t));
    keys = 0;
  }
  if (live) {
    const T* q = static_cast<const T*>(a.q) + orow;
    for (int c = lane; c < a.W; c += 32) qs[warp * a.W + c] = to_f32<T>(q[c]);
  }
  float acc[NC];
#pragma unroll
  for (int i = 0; i < NC; ++i) acc[i] = 0.0f;
  float m = -INFINITY, l = 0.0f;
  const T* cache = static_cast<const T*>(a.cache);
  for (int k0 = 0; k0 < keys; k0 += kKeys) {
    __syncthreads();
    for (int r = warp; r < kKeys; r += kWarps) {
      const int key = k0 + r;
      long long slot = -1;
      if (key < keys) {
        const int blk = a.block_tables[static_cast<long long>(pl.req) * a.max_blocks +
                                       key / a.block_size];
        slot = static_cast<long long>(blk) * a.block_size + key % a.block_size;
        if (slot < 0 || slot >= a.num_slots) {
          if (lane == 0)
            report_status(a.status, kStatusBounds, kKernelId + 2, static_cast<unsigned int>(t));
          slot = -1;
        }
      }
      for (int c = lane; c < a.W; c += 32)
        ks[r * pitch + c] = slot >= 0 ? to_f32<T>(cache[slot * a.W + c]) : 0.0f;
    }
    __syncthreads();
    if (!live) continue;
    float s = 0.0f;
    const float4* kr = reinterpret_cast<const float4*>(ks + lane * pitch);
    const float4* qr = reinterpret_cast<const float4*>(qs + warp * a.W);
    for (int c = 0; c < a.W / 4; ++c) {
      const float4 x = kr[c], y = qr[c];
      s += x.x * y.x + x.y * y.y + x.z * y.z + x.w * y.w;
    }
    s = k0 + lane < keys ? s * a.scale : -INFINITY;
    const float m_new = fmaxf(m, warp_max(s));       // finite: key k0 is visible
    const float p = expf(s - m_new);
    const float al = expf(m - m_new);
    l = l * al + warp_sum(p);
    m = m_new;
#pragma unroll
    for (int i = 0; i < NC; ++i) acc[i] *= al;
    const int nk = min(kKeys, keys - k0);
    for (int r = 0; r < nk; ++r) {
      const float pr = __shfl_sync(0xffffffffu, p, r);
      const float* kr1 = ks + r * pitch + lane;
#pragma unroll
      for (int i = 0; i < NC; ++i)
        if (i * 32 + lane < a.W) acc[i] += pr * kr1[i * 32];
    }
  }
  if (!live) return;
  float inv = 0.0f;
  if (l > 0.0f) {
    inv = 1.0f / l;
    if (a.sink != nullptr) {
      const float sink = a.sink[head], top = fmaxf(m, sink), f = expf(m - top);
      inv = f / (l * f + expf(sink - top));
    }
    if (a.gate != nullptr)
      inv /= 1.0f + expf(-to_f32<T>(static_cast<const T*>(a.gate)[t * a.ldg + head]));
  }
#pragma unroll
  for (int i = 0; i < NC; ++i)
    if (i * 32 + lane < a.W) out[orow + i * 32 + lane] = from_f32<T>(acc[i] * inv);
}

template <typename T, int NC>
static int launch_attention(const AttnArgs& a, cudaStream_t s) {
  const size_t smem = (static_cast<size_t>(kKeys) * key_pitch(a.W) +
                       static_cast<size_t>(kWarps) * a.W) * sizeof(float);
  if (smem > 220 * 1024) return -20;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(latent_attention_kernel<T, NC>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  dim3 grid(a.T, (a.N + kWarps - 1) / kWarps);
  latent_attention_kernel<T, NC><<<grid, kWarps * 32, smem, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int dispatch_attention(const AttnArgs& a, cudaStream_t s) {
  const int nc = (a.W + 31) / 32;
  if (nc <= 4) return launch_attention<T, 4>(a, s);
  if (nc <= 8) return launch_attention<T, 8>(a, s);
  if (nc <= 16) return launch_attention<T, 16>(a, s);
  if (nc <= 44) return launch_attention<T, 44>(a, s);
  return -20;
}

}  // namespace latent
}  // namespace b200

using namespace b200;
using namespace b200::latent;

// dtype (of kv, weight, cache, q and q_lat): 0 bf16, 2 fp32.  x / state null: no state rows.  R > 0:
// columns L .. L + R of kv are the key's rotated part and the last R of every head's dim + R columns
// of q the queries'; neighbours are rotated together.
B200_API int b200_latent_cache(const void* kv, long long ldkv, const void* weight, float eps,
                               void* cache, long long num_slots, int W, const long long* slots,
                               const float* x, float* state, const int* cu_q, int T, int L, int H,
                               int num_decodes, int num_prefills, int block_size, int R, int N,
                               int dim, const void* q, long long ldq, void* q_lat,
                               const float* cos_sin, long long max_pos, const long long* positions,
                               int dtype, void* stream) {
  if (T <= 0) return 0;
  if (L <= 0 || R < 0 || (R & 1) != 0 || W < L + R || block_size <= 0 || (dtype != 0 && dtype != 2) ||
      (R > 0 && (q == nullptr || q_lat == nullptr || cos_sin == nullptr || positions == nullptr ||
                 N <= 0 || dim < 0)))
    return -2;
  CacheArgs a;
  a.kv = kv; a.ldkv = ldkv; a.weight = weight; a.eps = eps; a.cache = cache;
  a.num_slots = num_slots; a.W = W; a.slots = slots; a.x = state ? x : nullptr; a.state = state;
  a.cu_q = cu_q; a.T = T; a.L = L; a.H = H; a.num_decodes = num_decodes;
  a.num_prefills = num_prefills; a.block_size = block_size; a.status = status_ptr();
  a.R = R; a.N = N; a.dim = dim; a.q = q; a.ldq = ldq; a.q_lat = q_lat; a.cos_sin = cos_sin;
  a.max_pos = max_pos; a.positions = positions;
  const auto even = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 3) == 0; };
  const bool pairs = (L & 1) == 0 && (dim & 1) == 0 && (W & 1) == 0 && (ldkv & 1) == 0 &&
                     (ldq & 1) == 0 && even(kv) && even(cache) && even(q) && even(q_lat);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 2) latent_cache_kernel<float, false><<<T, 128, 0, s>>>(a);
  else if (pairs) latent_cache_kernel<__nv_bfloat16, true><<<T, 128, 0, s>>>(a);
  else latent_cache_kernel<__nv_bfloat16, false><<<T, 128, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

// q / out [T, N, W], cache [num_slots, W], W a multiple of 4; -20: wider than the kernel covers.
// sink [N] and gate [T, ldg] (of q's type): optional.
B200_API int b200_latent_attention(const void* q, const void* cache, long long num_slots, void* out,
                                   const int* block_tables, int max_blocks, int block_size,
                                   const int* seq_lens, const int* cu_q, int T, int N, int W,
                                   int num_decodes, int num_prefills, float scale,
                                   const float* sink, const void* gate, long long ldg, int dtype,
                                   void* stream) {
  if (T <= 0 || N <= 0) return 0;
  if (W <= 0 || (W % 4) != 0 || block_size <= 0 || (dtype != 0 && dtype != 2)) return -2;
  AttnArgs a;
  a.q = q; a.cache = cache; a.num_slots = num_slots; a.out = out; a.block_tables = block_tables;
  a.max_blocks = max_blocks; a.block_size = block_size; a.seq_lens = seq_lens; a.cu_q = cu_q;
  a.T = T; a.N = N; a.W = W; a.num_decodes = num_decodes; a.num_prefills = num_prefills;
  a.scale = scale; a.sink = sink; a.gate = gate; a.ldg = ldg; a.status = status_ptr();
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == 0 ? dispatch_attention<__nv_bfloat16>(a, s) : dispatch_attention<float>(a, s);
}
