// Queries, keys and values of one step from a merged projection [q | k | v | ..] whose heads are normalised one by one:
//
//   q' = t(pos) N(R(pos) q),   k' = N(R(pos) k),   v' = v        (or R after N; R, t and the norm's weight are optional)
//
// N is an RMS norm over the dim channels of a head (and map), with a weight of dim channels shared by all heads or none;
// R turns pairs of the first `dims` channels: neighbours 2 i and 2 i + 1, or i and i + dims / 2; t is a factor per position.
// A head may have two maps, each with a query and a key of its own over one value: query rows lie side by side, map m's
// channels starting at m * q_shift of its row, and a key's maps share a cache row [map 1 | map 2].  Keys and values go to
// their paged caches, queries to rows the attention kernels read; every row is padded with zeros to its pitch.  Norms,
// angles and factors are 32-bit.  LPI lanes share one head of one token and move whole 16-byte groups where the sizes
// allow it.
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../common/launch.cuh"

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(__half v) { return __half2float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
template <> __device__ __forceinline__ __half from_f<__half>(float v) { return __float2half_rn(v); }

struct HeadParams {
  const void* proj;         // [T, ld]
  const float* wq;          // [dim] or null
  const float* wk;
  const int* positions;     // [T]
  const float* cos_sin;     // [max_pos, dims] rows [cos | sin] of dims / 2 frequencies, or null
  const float* factor;      // [max_pos] or null
  const int* slot_mapping;  // [T], < 0: no cache row
  void* q_out;              // [T, H * maps, qp]
  void* k_cache;            // [blocks, G, block_size, kp]
  void* v_cache;            // [blocks, G, block_size, vp]
  long ld, k_off, v_off;
  int T, H, G, maps, dim, vdim, dims, neighbours, weight_last, q_shift, qp, kp, vp, block_size, max_pos;
  float eps;
};

// V consecutive values (one 16-byte group, or a single value).
template <typename T, int V>
__device__ __forceinline__ void load_v(const T* p, float* x) {
  if constexpr (V == 1) {
    x[0] = to_f(*p);
  } else {
    alignas(16) T raw[V];
    *reinterpret_cast<uint4*>(raw) = *reinterpret_cast<const uint4*>(p);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = to_f(raw[e]);
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_v(T* p, const float* x) {
  if constexpr (V == 1) {
    *p = from_f<T>(x[0]);
  } else {
    alignas(16) T raw[V];
#pragma unroll
    for (int e = 0; e < V; ++e) raw[e] = from_f<T>(x[e]);
    *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(raw);
  }
}

// Weight of channel c (1 without one).
__device__ __forceinline__ float weight_at(const float* w, int c) { return w != nullptr ? w[c] : 1.f; }

template <typename T, int V, int LPI>
__global__ void __launch_bounds__(256) head_prepare_kernel(const HeadParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  const int nq = p.H * p.maps, nk = p.G * p.maps, per = nq + nk + p.G;
  const int sub = threadIdx.x % LPI;
  const long item = static_cast<long>(blockIdx.x) * (256 / LPI) + threadIdx.x / LPI;
  const bool live = item < static_cast<long>(p.T) * per;     // all lanes stay for the reductions
  const int t = live ? static_cast<int>(item / per) : 0, it = live ? static_cast<int>(item % per) : 0;
  const T* row = reinterpret_cast<const T*>(p.proj) + t * p.ld;
  const int slot = p.slot_mapping[t];
  const long blk = slot >= 0 ? slot / p.block_size : 0, off = slot >= 0 ? slot % p.block_size : 0;
  if (it >= nq + nk) {                                       // a value: copied (uniform over the lanes of an item)
    const int g = it - nq - nk;
    if (live && slot >= 0) {
      const T* src = row + p.v_off + static_cast<long>(g) * p.vdim;
      T* dst = reinterpret_cast<T*>(p.v_cache) + ((blk * p.G + g) * p.block_size + off) * p.vp;
      for (int c = sub * V; c < p.vp; c += LPI * V) {
        float x[V];
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = 0.f;
        if (c < p.vdim) load_v<T, V>(src + c, x);
        store_v<T, V>(dst + c, x);
      }
    }
  }
  const bool is_k = it >= nq && it < nq + nk, normed = it < nq + nk;
  const int h = is_k ? it - nq : it;
  const T* src = row + (is_k ? p.k_off : 0) + static_cast<long>(normed ? h : 0) * p.dim;
  float ss = 0.f;
  if (normed) {
    for (int c = sub * V; c < p.dim; c += LPI * V) {
      float x[V];
      load_v<T, V>(src + c, x);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(x[e], x[e], ss);
    }
  }
#pragma unroll
  for (int m = LPI / 2; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  if (!live || !normed || (is_k && slot < 0)) return;
  const int pos = min(max(p.positions[t], 0), p.max_pos - 1);
  float inv = 1.f / sqrtf(ss / static_cast<float>(p.dim) + p.eps);
  if (!is_k && p.factor != nullptr) inv *= p.factor[pos];
  const float* w = is_k ? p.wk : p.wq;
  const float* cs = p.cos_sin != nullptr ? p.cos_sin + static_cast<long>(pos) * p.dims : nullptr;
  const int half = p.dims / 2, map = h % p.maps;
  // destination row, the channels [lo, hi) of it that this item writes, and where its first channel lies
  T* dst;
  int lo = 0, hi, shift;
  if (is_k) {
    dst = reinterpret_cast<T*>(p.k_cache) + ((blk * p.G + h / p.maps) * p.block_size + off) * p.kp;
    shift = map * p.dim;
    lo = shift;
    hi = map + 1 == p.maps ? p.kp : shift + p.dim;
  } else {
    dst = reinterpret_cast<T*>(p.q_out) + (static_cast<long>(t) * nq + h) * p.qp;
    shift = map * p.q_shift;
    hi = p.qp;
  }
  for (int j = lo + sub * V; j < hi; j += LPI * V) {
    const int c = j - shift;
    float x[V], o[V];
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = 0.f;
    if (c >= 0 && c < p.dim) {
      load_v<T, V>(src + c, x);
      if (cs == nullptr || c >= p.dims) {
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = x[e] * inv * weight_at(w, c + e);
      } else if (p.neighbours) {
        // pairs lie inside a group; single values fetch their neighbour
        float y[V];
        if constexpr (V == 1) y[0] = to_f(src[c ^ 1]);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          if constexpr (V > 1) y[e] = x[e ^ 1];
          const int f = (c + e) >> 1;
          const float own = weight_at(w, c + e), ow = p.weight_last ? own : weight_at(w, (c + e) ^ 1);
          const float a = x[e] * own * cs[f], b = y[e] * ow * cs[half + f];
          o[e] = (((c + e) & 1) ? a + b : a - b) * inv;
        }
      } else {
        const bool first = c < half;
        const int other = first ? c + half : c - half;
        float y[V];
        load_v<T, V>(src + other, y);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const int f = first ? c + e : other + e;
          const float own = weight_at(w, c + e), ow = p.weight_last ? own : weight_at(w, other + e);
          const float a = x[e] * own * cs[f], b = y[e] * ow * cs[half + f];
          o[e] = (first ? a - b : a + b) * inv;
        }
      }
    }
    store_v<T, V>(dst + j, o);
  }
}

template <typename T, int V>
int launch(const HeadParams& p, cudaStream_t s) {
  const int per = p.H * p.maps + p.G * p.maps + p.G;
  int widest = p.qp > p.vp ? p.qp : p.vp;
  if (p.kp > widest) widest = p.kp;
  const int groups = (widest + V - 1) / V;
  const int lpi = groups <= 8 ? 8 : groups <= 16 ? 16 : 32;
  const long blocks = (static_cast<long>(p.T) * per * lpi + 255) / 256;
  if (blocks > 2147483647l) return -10;
  const dim3 grid(static_cast<unsigned>(blocks));
  if (lpi == 8) return static_cast<int>(fi::launch_kernel(head_prepare_kernel<T, V, 8>, grid, dim3(256), 0, s, 0, p));
  if (lpi == 16) return static_cast<int>(fi::launch_kernel(head_prepare_kernel<T, V, 16>, grid, dim3(256), 0, s, 0, p));
  return static_cast<int>(fi::launch_kernel(head_prepare_kernel<T, V, 32>, grid, dim3(256), 0, s, 0, p));
}

}  // namespace

// dtype: 0 bf16, 1 fp16, 2 fp32 (projection, queries, caches).  Slots >= 0 must lie inside the caches.  Columns of proj:
// q from 0 ([H, maps, dim]), k from k_off ([G, maps, dim]), v from v_off ([G, vdim]).  weight_last: the norm's weight
// multiplies what is already rotated.
extern "C" int fi_head_prepare(const void* proj, long ld, long k_off, long v_off, const float* wq, const float* wk, float eps,
                               const int* positions, const float* cos_sin, int dims, int neighbours, int weight_last,
                               const float* factor, int max_pos, const int* slot_mapping, void* q_out, int q_shift, int qp,
                               void* k_cache, int kp, void* v_cache, int vp, int T, int H, int G, int maps, int dim, int vdim,
                               int block_size, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || maps < 1 || dim <= 0 || vdim <= 0 || q_shift < 0 || qp < (maps - 1) * q_shift + dim ||
      kp < maps * dim || vp < vdim || block_size <= 0 || max_pos <= 0)
    return -10;
  if (cos_sin != nullptr && (dims < 0 || dims > dim || dims % 2 != 0)) return -10;
  HeadParams p = {};
  p.proj = proj; p.wq = wq; p.wk = wk; p.positions = positions; p.cos_sin = cos_sin; p.factor = factor;
  p.slot_mapping = slot_mapping; p.q_out = q_out; p.k_cache = k_cache; p.v_cache = v_cache; p.ld = ld; p.k_off = k_off;
  p.v_off = v_off; p.T = T; p.H = H; p.G = G; p.maps = maps; p.dim = dim; p.vdim = vdim;
  p.dims = cos_sin != nullptr ? dims : 0; p.neighbours = neighbours; p.weight_last = weight_last; p.q_shift = q_shift;
  p.qp = qp; p.kp = kp; p.vp = vp; p.block_size = block_size; p.max_pos = max_pos; p.eps = eps;
  const int v = dtype == 2 ? 4 : 8;
  const uintptr_t at = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q_out) |
                       reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache);
  const bool vec = ((dim | vdim | q_shift | qp | kp | vp) % v) == 0 && ld % v == 0 && k_off % v == 0 && v_off % v == 0 &&
                   p.dims % v == 0 && (neighbours || (p.dims / 2) % v == 0) && (at & 15) == 0;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (dtype == 0) return vec ? launch<__nv_bfloat16, 8>(p, s) : launch<__nv_bfloat16, 1>(p, s);
  if (dtype == 1) return vec ? launch<__half, 8>(p, s) : launch<__half, 1>(p, s);
  if (dtype == 2) return vec ? launch<float, 4>(p, s) : launch<float, 1>(p, s);
  return -11;
}
