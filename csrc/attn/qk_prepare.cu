// Queries, keys and values of one step from a merged projection [q (H * dim) | k (G * dim) | ..]:
//
//   q' = R(pos) rmsnorm(q) over all H * dim channels,   k' = R(pos) rmsnorm(k) over all G * dim channels,
//   v = k, or a projection of its own [.. | v (G * vdim)] whose channels 2 i and 2 i + 1 may turn by angle i of a second
//   table (over all vdim channels)
//
// Keys and values go to their paged caches, queries to rows the attention kernels read; heads are padded with zeros
// from dim to the kernels' head size.  The rotation turns channels i and i + dims / 2 of a head (i < dims / 2) by the
// angle of frequency i; cos_sin rows are [cos (dims / 2) | sin (dims / 2)]; channels from dims on pass.  Norms and angles
// are 32-bit.  One block per token: the sums of squares, then a second walk over the row (cached in L1) in whole
// 16-byte groups where the sizes allow it.
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

// N consecutive floats from a 16-byte boundary.
template <int N>
__device__ __forceinline__ void load_floats(const float* p, float* v) {
#pragma unroll
  for (int i = 0; i < N; i += 4) {
    const float4 f = *reinterpret_cast<const float4*>(p + i);
    v[i] = f.x; v[i + 1] = f.y; v[i + 2] = f.z; v[i + 3] = f.w;
  }
}

struct QkParams {
  const void* proj;         // [T, ld]
  const float* wq;          // [H * dim]
  const float* wk;          // [G * dim]
  const int* positions;     // [T]
  const float* cos_sin;     // [max_pos, dims]
  const int* slot_mapping;  // [T], < 0: no cache row
  void* q_out;              // [T, H, hd]
  void* k_cache;            // [blocks, G, block_size, hd]
  void* v_cache;
  long ld;
  int H, G, dim, hd, dims, block_size, max_pos;
  float eps;
  int v_off, vdim, vp;      // v_off > 0: values start there; vp: row pitch of the value cache
  const float* v_cs;        // [max_pos, vdim] or null
};

constexpr int kThreads = 128;

// VEC: every head, row and table starts on 16-byte groups.  A thread then keeps its place inside a head (and the angles of its
// channels) while it walks over heads.
template <typename T, bool VEC>
__global__ void __launch_bounds__(kThreads) qk_prepare_kernel(const QkParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  constexpr int V = 16 / sizeof(T);
  __shared__ float red[2][kThreads / 32];
  const int t = blockIdx.x, tid = threadIdx.x;
  const T* row = reinterpret_cast<const T*>(p.proj) + t * p.ld;
  const int nq = p.H * p.dim, nk = p.G * p.dim;
  const int per = VEC ? p.hd / V : p.hd;                   // groups (or channels) of a padded head
  const int step = VEC ? kThreads / per : 0;               // heads that the block handles at a time
  const int h0 = VEC ? tid / per : 0, c0 = VEC ? (tid - h0 * per) * V : 0;
  const bool mine = h0 < step && c0 < p.dim;
  const int pos = min(max(p.positions[t], 0), p.max_pos - 1), half = p.dims / 2, slot = p.slot_mapping[t];
  const float* cs = p.cos_sin + static_cast<long>(pos) * p.dims;
  float sq = 0.f, sk = 0.f;
  if constexpr (VEC) {
    if (mine) {
#pragma unroll 4
      for (int h = h0; h < p.H + p.G; h += step) {
        alignas(16) T x[V];
        *reinterpret_cast<uint4*>(x) = *reinterpret_cast<const uint4*>(row + h * p.dim + c0);
        float s = 0.f;
#pragma unroll
        for (int e = 0; e < V; ++e) { const float f = to_f(x[e]); s = fmaf(f, f, s); }
        if (h < p.H) sq += s; else sk += s;
      }
    }
  } else {
    for (int i = tid; i < nq + nk; i += kThreads) {
      const float f = to_f(row[i]);
      if (i < nq) sq = fmaf(f, f, sq); else sk = fmaf(f, f, sk);
    }
  }
  for (int m = 16; m > 0; m >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, m);
    sk += __shfl_xor_sync(0xffffffffu, sk, m);
  }
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < kThreads / 32; ++w) { sq += red[0][w]; sk += red[1][w]; }
  const float iq = 1.f / sqrtf(sq / static_cast<float>(nq) + p.eps), ik = 1.f / sqrtf(sk / static_cast<float>(nk) + p.eps);
  const int heads = slot >= 0 ? p.H + p.G : p.H;
  const int blk_i = slot >= 0 ? slot / p.block_size : 0;
  const long blk = blk_i, off = slot >= 0 ? slot - blk_i * p.block_size : 0;
  T* const q_out = reinterpret_cast<T*>(p.q_out) + static_cast<long>(t) * p.H * p.hd;
  if constexpr (VEC) {
    const bool turns = mine && c0 < p.dims, first = c0 < half;
    const int other = first ? c0 + half : c0 - half;
    float cc[V], ss[V];                                    // ss with the sign of the partner's share
#pragma unroll
    for (int e = 0; e < V; ++e) { cc[e] = 1.f; ss[e] = 0.f; }
    if (turns) {
      load_floats<V>(cs + (first ? c0 : other), cc);
      load_floats<V>(cs + half + (first ? c0 : other), ss);
      if (first)
#pragma unroll
        for (int e = 0; e < V; ++e) ss[e] = -ss[e];
    }
    if (h0 < step) {
#pragma unroll 4
      for (int h = h0; h < heads; h += step) {
        const bool is_k = h >= p.H;
        const int g = h - p.H;
        const long at = is_k ? ((blk * p.G + g) * p.block_size + off) * p.hd + c0 : 0;
        alignas(16) T x[V], o[V];
        *reinterpret_cast<uint4*>(x) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(o) = make_uint4(0, 0, 0, 0);
        if (mine) {
          const T* src = row + h * p.dim;                  // heads of k follow those of q
          const float* w = is_k ? p.wk + g * p.dim : p.wq + h * p.dim;
          const float inv = is_k ? ik : iq;
          float wx[V], a[V];
          *reinterpret_cast<uint4*>(x) = *reinterpret_cast<const uint4*>(src + c0);
          load_floats<V>(w + c0, wx);
#pragma unroll
          for (int e = 0; e < V; ++e) a[e] = to_f(x[e]) * inv * wx[e];
          if (turns) {
            alignas(16) T y[V];
            *reinterpret_cast<uint4*>(y) = *reinterpret_cast<const uint4*>(src + other);
            load_floats<V>(w + other, wx);
#pragma unroll
            for (int e = 0; e < V; ++e) a[e] = fmaf(a[e], cc[e], to_f(y[e]) * inv * wx[e] * ss[e]);
          }
#pragma unroll
          for (int e = 0; e < V; ++e) o[e] = from_f<T>(a[e]);
        }
        if (is_k) {
          *reinterpret_cast<uint4*>(reinterpret_cast<T*>(p.k_cache) + at) = *reinterpret_cast<const uint4*>(o);
          if (p.v_off == 0) *reinterpret_cast<uint4*>(reinterpret_cast<T*>(p.v_cache) + at) = *reinterpret_cast<const uint4*>(x);
        } else {
          *reinterpret_cast<uint4*>(q_out + h * p.hd + c0) = *reinterpret_cast<const uint4*>(o);
        }
      }
    }
  } else {
    for (int i = tid; i < heads * per; i += kThreads) {
      const int h = i / per, c = i % per;
      const bool is_k = h >= p.H;
      const T* src = row + h * p.dim;
      const float* w = is_k ? p.wk + (h - p.H) * p.dim : p.wq + h * p.dim;
      const float inv = is_k ? ik : iq;
      const long at = is_k ? ((blk * p.G + h - p.H) * p.block_size + off) * p.hd + c : 0;
      T x = from_f<T>(0.f);
      float a = 0.f;
      if (c < p.dim) {
        x = src[c];
        a = to_f(x) * inv * w[c];
        if (c < p.dims) {
          const bool first = c < half;
          const int other = first ? c + half : c - half, f = first ? c : other;
          const float bb = to_f(src[other]) * inv * w[other];
          a = first ? a * cs[f] - bb * cs[half + f] : a * cs[f] + bb * cs[half + f];
        }
      }
      if (is_k) {
        reinterpret_cast<T*>(p.k_cache)[at] = from_f<T>(a);
        if (p.v_off == 0) reinterpret_cast<T*>(p.v_cache)[at] = x;
      } else {
        q_out[h * p.hd + c] = from_f<T>(a);
      }
    }
  }
  if (p.v_off == 0 || slot < 0) return;
  const float* vcs = p.v_cs != nullptr ? p.v_cs + static_cast<long>(pos) * p.vdim : nullptr;
  T* v0 = reinterpret_cast<T*>(p.v_cache);
  if constexpr (VEC) {
    const int vper = p.vp / V;
    for (int i = tid; i < p.G * vper; i += kThreads) {
      const int g = i / vper, c = (i % vper) * V;
      alignas(16) T x[V];
      *reinterpret_cast<uint4*>(x) = make_uint4(0, 0, 0, 0);
      if (c < p.vdim) {
        *reinterpret_cast<uint4*>(x) = *reinterpret_cast<const uint4*>(row + p.v_off + g * p.vdim + c);
        if (vcs != nullptr) {
          float cc[V / 2], ss[V / 2];
          if constexpr (V == 8) {
            load_floats<V / 2>(vcs + c / 2, cc);
            load_floats<V / 2>(vcs + (p.vdim + c) / 2, ss);
          } else {
#pragma unroll
            for (int e = 0; e < V / 2; ++e) { cc[e] = vcs[c / 2 + e]; ss[e] = vcs[(p.vdim + c) / 2 + e]; }
          }
#pragma unroll
          for (int e = 0; e < V; e += 2) {
            const float a = to_f(x[e]), bb = to_f(x[e + 1]);
            x[e] = from_f<T>(a * cc[e / 2] - bb * ss[e / 2]);
            x[e + 1] = from_f<T>(bb * cc[e / 2] + a * ss[e / 2]);
          }
        }
      }
      *reinterpret_cast<uint4*>(v0 + ((blk * p.G + g) * p.block_size + off) * p.vp + c) = *reinterpret_cast<const uint4*>(x);
    }
  } else {
    for (int i = tid; i < p.G * p.vp; i += kThreads) {
      const int g = i / p.vp, c = i % p.vp;
      float a = 0.f;
      if (c < p.vdim) {
        const T* src = row + p.v_off + g * p.vdim;
        a = to_f(src[c]);
        if (vcs != nullptr) {
          const float bb = to_f(src[c ^ 1]), cc = vcs[c / 2], ss = vcs[p.vdim / 2 + c / 2];
          a = c & 1 ? a * cc + bb * ss : a * cc - bb * ss;
        }
      }
      v0[((blk * p.G + g) * p.block_size + off) * p.vp + c] = from_f<T>(a);
    }
  }
}

template <typename T>
int launch(const QkParams& p, bool vec, int tokens, cudaStream_t s) {
  return static_cast<int>(fi::launch_kernel(vec ? qk_prepare_kernel<T, true> : qk_prepare_kernel<T, false>, dim3(tokens), dim3(kThreads), 0, s, 0, p));
}

}  // namespace

// dtype: 0 bf16, 1 fp16, 2 fp32 (projection, queries, caches).  Slots >= 0 must lie inside the caches.  v_off 0: the value is
// the key's projection (vdim, vp and v_cs unused); otherwise values are G heads of vdim channels from column v_off on, in
// cache rows of vp channels, turned by v_cs [max_pos, vdim] unless that is null.
extern "C" int fi_qk_prepare(const void* proj, long ld, const float* wq, const float* wk, float eps, const int* positions,
                             const float* cos_sin, int max_pos, const int* slot_mapping, void* q_out, void* k_cache,
                             void* v_cache, int T, int H, int G, int dim, int hd, int dims, int block_size, int v_off, int vdim,
                             int vp, const float* v_cs, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || dim <= 0 || hd < dim || dims < 0 || dims > dim || dims % 2 != 0 || block_size <= 0 || max_pos <= 0)
    return -10;
  if (v_off != 0 && (v_off < (H + G) * dim || vdim <= 0 || vp < vdim || (v_cs != nullptr && vdim % 2 != 0))) return -10;
  QkParams p = {};
  p.v_off = v_off; p.vdim = vdim; p.vp = vp; p.v_cs = v_cs;
  p.proj = proj; p.wq = wq; p.wk = wk; p.positions = positions; p.cos_sin = cos_sin; p.slot_mapping = slot_mapping;
  p.q_out = q_out; p.k_cache = k_cache; p.v_cache = v_cache; p.ld = ld; p.H = H; p.G = G; p.dim = dim; p.hd = hd;
  p.dims = dims; p.block_size = block_size; p.max_pos = max_pos; p.eps = eps;
  const int v = dtype == 2 ? 4 : 8;
  const uintptr_t at = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q_out) | reinterpret_cast<uintptr_t>(wq) |
                       reinterpret_cast<uintptr_t>(wk) | reinterpret_cast<uintptr_t>(cos_sin) | reinterpret_cast<uintptr_t>(v_cs) |
                       reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache);
  const bool vec = dim % v == 0 && hd / v <= kThreads && hd % v == 0 && (dims / 2) % v == 0 && ld % v == 0 && (at & 15) == 0 &&
          (v_off == 0 || (v_off % v == 0 && vdim % v == 0 && vp % v == 0));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (dtype == 0) return launch<__nv_bfloat16>(p, vec, T, s);
  if (dtype == 1) return launch<__half>(p, vec, T, s);
  if (dtype == 2) return launch<float>(p, vec, T, s);
  return -11;
}
