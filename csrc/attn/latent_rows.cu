// Helpers around latent attention (one shared cache row per token, [RMS-normed latent | rotary key]) for any head
// geometry, and a general attention kernel over such rows in 32-bit arithmetic.
//
//   latent_prepare_kernel   per token: norm of the latent + rotation of the shared key -> cache row; rotation of every
//                           head's rotary query part into the caller's query layout
//   latent_gather_kernel    cache rows of a list of slots -> contiguous latents (what the per-head up-projections read)
//   latent_pool_kernel      up-projected keys and values + the cached rotary keys -> padded per-head K / V tiles of a
//                           temporary pool that the prefill attention kernels read
//   latent_rows_kernel      a warp per (row, head): scores against the cache rows, softmax with window and sink, sum of
//                           latents (or of the rows of a value cache, with grouped heads and an output gate).  Runs
//                           32-bit models and geometries outside the tensor-core kernels.
// Rotation pairs are neighbours: channels (2i, 2i + 1) turn by the angle of frequency i; cos_sin rows are
// [cos(dims / 2) | sin(dims / 2)].  Positions, angles, norms, scores and weights are 32-bit.
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <math_constants.h>
#include <stdint.h>

#include "../common/launch.cuh"
#include "attn_extra.h"

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(__half v) { return __half2float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
template <> __device__ __forceinline__ __half from_f<__half>(float v) { return __float2half_rn(v); }

struct PrepareParams {
  const void* q;            // [T, ldq]: head h at h * (dim + rot), rotary part last
  const void* dkv;          // [T, ldkv]: latent (rank) then rotary key (rot)
  const float* norm_w;      // [rank]
  const int* positions;     // [T]
  const float* cos_sin;     // [max_pos, rdims]
  const int* slot_mapping;  // [T], < 0: no cache row
  void* cache;              // rows of rank + rot values
  void* q_out;              // [T, nh, q_pitch]
  long ldq, ldkv;
  int T, nh, dim, rot, rdims, rank, q_pitch, nope_off, rot_off, zero_from, max_pos;
  int pairs, vec;           // alignment of all rows and parts: whole pairs, whole 16-byte groups
  int chunks;               // > 0: 16-byte groups written per head (all parts aligned)
  float eps;
};

// Values are handled in pairs: a pair of 16-bit values is one 32-bit access, and a rotation turns exactly one pair.
template <typename T> struct Pair;
template <> struct Pair<float> { typedef float2 type; };
template <> struct Pair<__nv_bfloat16> { typedef __nv_bfloat162 type; };
template <> struct Pair<__half> { typedef __half2 type; };
template <typename T> __device__ __forceinline__ float2 load_pair(const T* p, bool whole) {
  float2 r;
  if (whole) {
    const typename Pair<T>::type v = *reinterpret_cast<const typename Pair<T>::type*>(p);
    r.x = to_f(v.x); r.y = to_f(v.y);
  } else {
    r.x = to_f(p[0]); r.y = to_f(p[1]);
  }
  return r;
}
template <typename T> __device__ __forceinline__ void store_pair(T* p, float a, float b, bool whole) {
  if (whole) {
    typename Pair<T>::type v;
    v.x = from_f<T>(a); v.y = from_f<T>(b);
    *reinterpret_cast<typename Pair<T>::type*>(p) = v;
  } else {
    p[0] = from_f<T>(a); p[1] = from_f<T>(b);
  }
}

// Block: (token, share of the heads).  The first block of a token also writes its cache row.
template <typename T>
__global__ void __launch_bounds__(128) latent_prepare_kernel(const PrepareParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  __shared__ float red[4];
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = min(max(p.positions[t], 0), p.max_pos - 1);
  const float* cs = p.cos_sin + static_cast<long>(pos) * p.rdims;
  const int half = p.rdims / 2;
  const T* q = reinterpret_cast<const T*>(p.q) + t * p.ldq;
  const bool even = p.pairs != 0;                  // every row and every part of it starts on a whole pair
  // pair i of a rotary part of `n` channels (the last one may be half a pair, which never turns)
  auto turn = [&](const T* src, T* dst, int i, int n) {
    if (2 * i + 1 < n) {
      float2 v = load_pair(src + 2 * i, even);
      if (i < half) {
        const float c = cs[i], s = cs[half + i];
        v = make_float2(v.x * c - v.y * s, v.y * c + v.x * s);
      }
      store_pair(dst + 2 * i, v.x, v.y, even);
    } else {
      dst[2 * i] = src[2 * i];
    }
  };
  if (blockIdx.y == 0) {
    const T* row = reinterpret_cast<const T*>(p.dkv) + t * p.ldkv;
    float ss = 0.f;
    if (even) {
      for (int i = threadIdx.x; i < p.rank / 2; i += 128) {
        const float2 f = load_pair(row + 2 * i, true);
        ss += f.x * f.x + f.y * f.y;
      }
    } else {
      for (int i = threadIdx.x; i < p.rank; i += 128) { const float f = to_f(row[i]); ss += f * f; }
    }
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    const float inv = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / static_cast<float>(p.rank) + p.eps);
    const int slot = p.slot_mapping[t];
    if (slot >= 0) {
      T* dst = reinterpret_cast<T*>(p.cache) + static_cast<long>(slot) * (p.rank + p.rot);
      if (even) {
        for (int i = threadIdx.x; i < p.rank / 2; i += 128) {
          const float2 f = load_pair(row + 2 * i, true);
          store_pair(dst + 2 * i, f.x * inv * p.norm_w[2 * i], f.y * inv * p.norm_w[2 * i + 1], true);
        }
      } else {
        for (int i = threadIdx.x; i < p.rank; i += 128) dst[i] = from_f<T>(to_f(row[i]) * inv * p.norm_w[i]);
      }
      for (int i = threadIdx.x; i < (p.rot + 1) / 2; i += 128) turn(row + p.rank, dst + p.rank, i, p.rot);
    }
  }
  const int hd = p.dim + p.rot;
  constexpr int V = 16 / sizeof(T);
  if (p.chunks > 0) {
    // everything starts on 16-byte groups: a thread takes whole groups of all heads (copied, turned or cleared);
    // `chunks` groups per head are written, starting at group 0 of the query or at its rotary part
    const int total = p.nh * p.chunks, step = 128 * gridDim.y;
    const int first = p.nope_off >= 0 ? 0 : p.dim;
#pragma unroll 2
    for (int i = blockIdx.y * 128 + threadIdx.x; i < total; i += step) {
      const int h = i / p.chunks, c = first + (i % p.chunks) * V;
      T* dst = reinterpret_cast<T*>(p.q_out) + (static_cast<long>(t) * p.nh + h) * p.q_pitch +
               (c >= p.dim ? c - p.dim + p.rot_off : c + p.nope_off);
      uint4 raw = make_uint4(0, 0, 0, 0);
      if (c < hd) raw = *reinterpret_cast<const uint4*>(q + static_cast<long>(h) * hd + c);
      if (c >= p.dim && c < hd) {
        alignas(16) typename Pair<T>::type v[V / 2];
        *reinterpret_cast<uint4*>(v) = raw;
#pragma unroll
        for (int e = 0; e < V / 2; ++e) {
          const int pr = (c - p.dim) / 2 + e;
          if (pr < half) {
            const float x = to_f(v[e].x), y = to_f(v[e].y), cc = cs[pr], ss = cs[half + pr];
            v[e].x = from_f<T>(x * cc - y * ss);
            v[e].y = from_f<T>(y * cc + x * ss);
          }
        }
        raw = *reinterpret_cast<const uint4*>(v);
      }
      *reinterpret_cast<uint4*>(dst) = raw;
    }
    return;
  }
  for (int h = blockIdx.y * 4 + warp; h < p.nh; h += 4 * gridDim.y) {
    const T* src = q + static_cast<long>(h) * hd;
    T* dst = reinterpret_cast<T*>(p.q_out) + (static_cast<long>(t) * p.nh + h) * p.q_pitch;
    for (int i = lane; i < (p.rot + 1) / 2; i += 32) turn(src + p.dim, dst + p.rot_off, i, p.rot);
    if (p.nope_off >= 0) {
      if (p.vec) {
        for (int i = lane; i < p.dim / V; i += 32)
          reinterpret_cast<uint4*>(dst + p.nope_off)[i] = reinterpret_cast<const uint4*>(src)[i];
      } else {
        for (int i = lane; i < p.dim; i += 32) dst[p.nope_off + i] = src[i];
      }
      for (int i = p.zero_from + lane; i < p.q_pitch; i += 32) dst[i] = from_f<T>(0.f);
    }
  }
}

// out [n, pitch] (values beyond rank stay zero) from the cache rows of slots[i]; a negative slot gives a zero row.
template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const T* __restrict__ cache, const int* __restrict__ slots,
                                                            T* __restrict__ out, int n, int rank, int kd, int pitch,
                                                            int num_rows) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  constexpr int V = 16 / sizeof(T);
  const int per = (pitch + V - 1) / V;
  const bool vec = rank % V == 0 && kd % V == 0 && pitch % V == 0;
  for (long i = static_cast<long>(blockIdx.x) * 256 + threadIdx.x; i < static_cast<long>(n) * per;
       i += static_cast<long>(gridDim.x) * 256) {
    const int r = static_cast<int>(i / per), c = static_cast<int>(i % per) * V;
    const int slot = slots[r];
    const bool ok = slot >= 0 && slot < num_rows;
    if (vec) {
      uint4 v = make_uint4(0, 0, 0, 0);
      if (ok && c < rank) v = *reinterpret_cast<const uint4*>(cache + static_cast<long>(slot) * kd + c);
      *reinterpret_cast<uint4*>(out + static_cast<long>(r) * pitch + c) = v;
    } else {
      for (int e = c; e < min(c + V, pitch); ++e)
        out[static_cast<long>(r) * pitch + e] = (ok && e < rank) ? cache[static_cast<long>(slot) * kd + e] : from_f<T>(0.f);
    }
  }
}

// Row i of the step's context (block i / 128, row i % 128 of the temporary pool [n / 128, nh, 128, hd]):
// K = [key (dim) | cached rotary key (rot) | 0], V = [value (vdim) | 0]; rows with a negative slot are zero.
template <typename T>
__global__ void __launch_bounds__(256) latent_pool_kernel(const T* __restrict__ cache, const int* __restrict__ slots,
                                                          const T* __restrict__ kv, long ldkv, T* __restrict__ k_pool,
                                                          T* __restrict__ v_pool, int nh, int dim, int rot, int vdim,
                                                          int rank, int hd, int num_rows) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  constexpr int BS = 128;
  const int r = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slot = slots[r];
  const bool ok = slot >= 0 && slot < num_rows;
  const T* krow = kv + static_cast<long>(r) * ldkv;
  const T* vrow = krow + static_cast<long>(nh) * dim;
  const T* rrow = cache + static_cast<long>(ok ? slot : 0) * (rank + rot) + rank;
  const bool vec = ((dim | rot | vdim | rank) & 7) == 0 && (ldkv & 7) == 0;
  if (vec) {
    // hd / 8 groups of K and as many of V per head, spread over the block
    const int per = hd / 4, total = nh * per;
    const long row0 = (static_cast<long>(r / BS) * nh * BS + r % BS) * hd;
#pragma unroll 4
    for (int i = blockIdx.y * 256 + threadIdx.x; i < total; i += 256 * gridDim.y) {
      const int h = i / per, c8 = i % per;
      const bool is_v = c8 >= hd / 8;
      const int c = (is_v ? c8 - hd / 8 : c8) * 8;
      const T* src = nullptr;
      if (ok) {
        if (is_v) src = c < vdim ? vrow + static_cast<long>(h) * vdim + c : nullptr;
        else src = c < dim ? krow + static_cast<long>(h) * dim + c : (c < dim + rot ? rrow + c - dim : nullptr);
      }
      uint4 v = make_uint4(0, 0, 0, 0);
      if (src != nullptr) v = *reinterpret_cast<const uint4*>(src);
      *reinterpret_cast<uint4*>((is_v ? v_pool : k_pool) + row0 + static_cast<long>(h) * BS * hd + c) = v;
    }
    return;
  }
  for (int h = blockIdx.y * 8 + warp; h < nh; h += 8 * gridDim.y) {
    const long dst = ((static_cast<long>(r / BS) * nh + h) * BS + r % BS) * hd;
    for (int c8 = lane; c8 < hd / 4; c8 += 32) {        // hd / 8 chunks of K, then of V
      const bool is_v = c8 >= hd / 8;
      const int c = (is_v ? c8 - hd / 8 : c8) * 8;
      T* out = (is_v ? v_pool : k_pool) + dst + c;
        for (int e = 0; e < 8; ++e) {
          T v = from_f<T>(0.f);
          if (ok) {
            if (is_v) {
              if (c + e < vdim) v = vrow[static_cast<long>(h) * vdim + c + e];
            } else if (c + e < dim) {
              v = krow[static_cast<long>(h) * dim + c + e];
            } else if (c + e < dim + rot) {
              v = rrow[c + e - dim];
            }
          }
          out[e] = v;
        }
    }
  }
}

struct RowsParams {
  const void* q_cat;        // [rows, nh, kd / maps]
  const void* cache;        // [blocks, nkv, block size] rows of kd values
  const void* v_cache;      // the same with rows of vd values; null: the first vd values of a cache row are the value
  int nkv;
  void* out;                // element (row r, output head h, d) at out + h * out_head_stride + r * out_row_stride + d
  long out_head_stride, out_row_stride;
  const int* block_tables;
  const int* row_lens;
  const int* seq_of_row;    // or null
  int rows, nh, kd, vd, max_blocks, block_size, window, num_rows;
  float sm_scale;
  FiAttnExtra x;            // sinks, output gate, two maps per head (the key row of a head is [map 1 | map 2])
};

template <typename T, int NV, int MAPS, bool SIG>
__global__ void __launch_bounds__(128) latent_rows_kernel(const RowsParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  extern __shared__ float smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long item = static_cast<long>(blockIdx.x) * 4 + warp;
  const int heads = p.nh / MAPS, qd = p.kd / MAPS;
  if (item >= static_cast<long>(p.rows) * heads) return;
  const int r = static_cast<int>(item / heads), h = static_cast<int>(item % heads);
  float* q = smem + warp * p.kd;
  const T* qs = reinterpret_cast<const T*>(p.q_cat) + item * p.kd;      // a head's maps follow one another
  for (int i = lane; i < p.kd; i += 32) q[i] = to_f(qs[i]) * p.sm_scale;
  __syncwarp();
  const int len = min(p.row_lens[r], p.max_blocks * p.block_size);
  const int lo = SIG ? fi::first_key(p, max(0, len - 1)) : (p.window > 0 ? max(0, len - p.window) : 0);
  const int* bt = p.block_tables + static_cast<long>(p.seq_of_row ? p.seq_of_row[r] : r) * p.max_blocks;
  const T* cache = reinterpret_cast<const T*>(p.cache);
  const T* values = reinterpret_cast<const T*>(p.v_cache != nullptr ? p.v_cache : p.cache);
  const int vpitch = p.v_cache != nullptr ? p.vd : p.kd, kvh = h / (heads / p.nkv);
  float first[MAPS == 2 ? NV : 1];       // the first map's output
  float o[NV];
  for (int map = 0; map < MAPS; ++map) {
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i] = 0.f;
    float m = -CUDART_INF_F, l = 0.f;
    for (int k0 = lo; k0 < len; k0 += 32) {
      const int tok = k0 + lane;
      long src = 0;
      float s = -CUDART_INF_F;
      if (tok < len) {
        long blk = bt[tok / p.block_size];
        blk = blk < 0 || (blk + 1) * p.block_size > p.num_rows ? 0 : blk;
        src = (blk * p.nkv + kvh) * p.block_size + tok % p.block_size;
        const T* row = cache + src * p.kd + map * qd;
        const float* qm = q + map * qd;
        float a0 = 0.f, a1 = 0.f;
        int i = 0;
        for (; i + 1 < qd; i += 2) { a0 = fmaf(qm[i], to_f(row[i]), a0); a1 = fmaf(qm[i + 1], to_f(row[i + 1]), a1); }
        if (i < qd) a0 = fmaf(qm[i], to_f(row[i]), a0);
        s = a0 + a1;
      }
      float pv;
      if constexpr (SIG) {
        pv = tok < len ? 1.f / (1.f + __expf(-(s + p.x.bias[h]))) : 0.f;
      } else {
        float mx = s;
        for (int x = 16; x > 0; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
        const float nm = fmaxf(m, mx);            // at least one key of the chunk is visible
        const float alpha = __expf(m - nm);
        pv = __expf(s - nm);
        float rs = pv;
        for (int x = 16; x > 0; x >>= 1) rs += __shfl_xor_sync(0xffffffffu, rs, x);
        l = l * alpha + rs;
        m = nm;
#pragma unroll
        for (int i = 0; i < NV; ++i) o[i] *= alpha;
      }
      const int n = min(32, len - k0);
      for (int j = 0; j < n; ++j) {
        const float pj = __shfl_sync(0xffffffffu, pv, j);
        const T* row = values + __shfl_sync(0xffffffffu, src, j) * vpitch;
#pragma unroll
        for (int i = 0; i < NV; ++i)
          if (i * 32 + lane < p.vd) o[i] = fmaf(pj, to_f(row[i * 32 + lane]), o[i]);
      }
    }
    if (p.x.sinks != nullptr && m != -CUDART_INF_F) l += __expf(p.x.sinks[h * MAPS + map] - m);
    const float inv = SIG ? 1.f : (l > 0.f ? 1.f / l : 0.f);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      o[i] *= inv;
      if constexpr (MAPS == 2) {
        if (map == 0) first[i] = o[i];
      }
    }
  }
  if constexpr (MAPS == 2) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      o[i] = first[i] - p.x.lambda * o[i];       // channels from vd on are zero
      ss = fmaf(o[i], o[i], ss);
    }
    for (int x = 16; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    const float f = p.x.out_scale / sqrtf(ss / static_cast<float>(p.vd) + p.x.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) o[i] *= f;
  }
  T* out = reinterpret_cast<T*>(p.out) + h * p.out_head_stride + r * p.out_row_stride;
  if constexpr (SIG) {
    if (p.x.turn != nullptr) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {           // neighbouring lanes hold the two channels of a pair
        const float other = __shfl_xor_sync(0xffffffffu, o[i], 1);
        const int d = i * 32 + lane;
        if (d < p.vd) {
          float u = lane & 1 ? other : o[i], v = lane & 1 ? o[i] : other;
          fi::turn_back(p, len - 1, d >> 1, u, v);
          o[i] = lane & 1 ? v : u;
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (i * 32 + lane < p.vd) {
      float v = o[i];
      if (p.x.gate != nullptr) {
        const long at = r * p.x.gate_stride + (p.x.gate_per_head ? h : h * p.vd + i * 32 + lane);
        v /= 1.f + __expf(-to_f(reinterpret_cast<const T*>(p.x.gate)[at]));
      }
      out[i * 32 + lane] = from_f<T>(v);
    }
}

template <typename T>
int launch_rows(const RowsParams& p, cudaStream_t s) {
  const long items = static_cast<long>(p.rows) * (p.nh / p.x.maps);
  const dim3 grid(static_cast<unsigned>((items + 3) / 4));
  const int smem = 4 * p.kd * 4;
#define FI_ROWS(N)                                                                                                         \
  return static_cast<int>(p.x.bias != nullptr ? fi::launch_kernel(latent_rows_kernel<T, N, 1, true>, grid, dim3(128), smem, s, 0, p) \
                          : p.x.maps == 2 ? fi::launch_kernel(latent_rows_kernel<T, N, 2, false>, grid, dim3(128), smem, s, 0, p)    \
                                          : fi::launch_kernel(latent_rows_kernel<T, N, 1, false>, grid, dim3(128), smem, s, 0, p))
  if (p.vd <= 64) FI_ROWS(2);
  if (p.vd <= 128) FI_ROWS(4);
  if (p.vd <= 256) FI_ROWS(8);
  if (p.vd <= 512) FI_ROWS(16);
  FI_ROWS(32);
#undef FI_ROWS
}

}  // namespace

#define FI_BY_TYPE(dtype, CALL)                 \
  if (dtype == 0) { CALL(__nv_bfloat16); }      \
  else if (dtype == 1) { CALL(__half); }        \
  else if (dtype == 2) { CALL(float); }         \
  else return -11;

// dtype: 0 bf16, 1 fp16, 2 fp32 (q, dkv, cache, q_out).  nope_off < 0: only the rotary parts of the queries are
// written; otherwise the other dimensions are copied to nope_off and [zero_from, q_pitch) is cleared.
extern "C" int fi_latent_prepare(const void* q, long ldq, const void* dkv, long ldkv, const float* norm_w, float eps,
                                 const int* positions, const float* cos_sin, int max_pos, const int* slot_mapping,
                                 void* cache, void* q_out, int q_pitch, int nope_off, int rot_off, int zero_from, int T,
                                 int nh, int dim, int rot, int rdims, int rank, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (nh <= 0 || dim < 0 || rot < 0 || rank <= 0 || rdims < 0 || rdims > rot || rdims % 2 != 0 || max_pos <= 0 ||
      rot_off < 0 || rot_off + rot > q_pitch || (nope_off >= 0 && (nope_off + dim > q_pitch || zero_from < 0)))
    return -10;
  PrepareParams p = {};
  p.q = q; p.dkv = dkv; p.norm_w = norm_w; p.positions = positions; p.cos_sin = cos_sin; p.slot_mapping = slot_mapping;
  p.cache = cache; p.q_out = q_out; p.ldq = ldq; p.ldkv = ldkv; p.T = T; p.nh = nh; p.dim = dim; p.rot = rot;
  p.rdims = rdims; p.rank = rank; p.q_pitch = q_pitch; p.nope_off = nope_off; p.rot_off = rot_off;
  p.zero_from = zero_from; p.max_pos = max_pos; p.eps = eps;
  const int esz = dtype == 2 ? 4 : 2, v = 16 / esz;
  const uintptr_t at = reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(dkv) | reinterpret_cast<uintptr_t>(cache) |
                       reinterpret_cast<uintptr_t>(q_out);
  p.pairs = ((ldq | ldkv | dim | rot | rank | q_pitch | rot_off) & 1) == 0 && (at & (2 * esz - 1)) == 0;
  p.vec = nope_off >= 0 && ldq % v == 0 && (dim + rot) % v == 0 && dim % v == 0 && q_pitch % v == 0 && nope_off % v == 0 &&
          ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(q_out)) & 15) == 0;
  const bool groups = ((dim | rot | q_pitch | rot_off) % v) == 0 && ldq % v == 0 &&
                      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(q_out)) & 15) == 0;
  if (groups && nope_off < 0) p.chunks = rot / v;
  // parts in the order [other dimensions | rotary part | cleared]
  if (groups && nope_off == 0 && rot_off == dim && zero_from == dim + rot) p.chunks = q_pitch / v;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(T, T >= 256 ? 1 : (nh + 3) / 4);
#define FI_CALL(TT) return static_cast<int>(fi::launch_kernel(latent_prepare_kernel<TT>, grid, dim3(128), 0, s, 0, p))
  FI_BY_TYPE(dtype, FI_CALL)
#undef FI_CALL
  return 0;
}

// out [n, pitch] of dtype; cache holds num_rows rows of kd values.
extern "C" int fi_latent_gather(const void* cache, const int* slots, void* out, int n, int rank, int kd, int pitch,
                                int num_rows, int dtype, void* stream) {
  if (n <= 0) return 0;
  if (rank <= 0 || kd < rank || pitch < rank || num_rows <= 0 || (reinterpret_cast<uintptr_t>(out) & 15) != 0 ||
      (reinterpret_cast<uintptr_t>(cache) & 15) != 0)
    return -10;
  const long work = static_cast<long>(n) * ((pitch + 3) / 4);
  const unsigned grid = static_cast<unsigned>(work / 256 + 1 < 1184 ? work / 256 + 1 : 1184);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define FI_CALL(TT) return static_cast<int>(fi::launch_kernel(latent_gather_kernel<TT>, dim3(grid), dim3(256), 0, s, 0, \
    (const TT*)cache, slots, (TT*)out, n, rank, kd, pitch, num_rows))
  FI_BY_TYPE(dtype, FI_CALL)
#undef FI_CALL
  return 0;
}

// n (a multiple of 128) context rows -> pools [n / 128, nh, 128, hd]; kv: [n, ldkv] = [nh * dim | nh * vdim].
extern "C" int fi_latent_pool(const void* cache, const int* slots, const void* kv, long ldkv, void* k_pool, void* v_pool,
                              int n, int nh, int dim, int rot, int vdim, int rank, int hd, int num_rows, int dtype,
                              void* stream) {
  if (n <= 0) return 0;
  if (n % 128 != 0 || nh <= 0 || dim + rot > hd || vdim > hd || hd % 8 != 0 || num_rows <= 0) return -10;
  if ((reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(k_pool) | reinterpret_cast<uintptr_t>(v_pool) |
       reinterpret_cast<uintptr_t>(cache)) & 15)
    return -10;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(n, n >= 1024 ? 1 : (nh + 7) / 8);
#define FI_CALL(TT) return static_cast<int>(fi::launch_kernel(latent_pool_kernel<TT>, grid, dim3(256), 0, s, 0, \
    (const TT*)cache, slots, (const TT*)kv, ldkv, (TT*)k_pool, (TT*)v_pool, nh, dim, rot, vdim, rank, hd, num_rows))
  if (dtype == 0) { FI_CALL(__nv_bfloat16); }
  if (dtype == 1) { FI_CALL(__half); }
#undef FI_CALL
  return -11;
}

// General attention of flattened rows over latent cache rows, 32-bit arithmetic.  window <= 0: none; sinks may be null.
extern "C" int fi_latent_rows(const void* q_cat, const void* cache, void* out, long out_head_stride, long out_row_stride,
                              const int* block_tables, const int* row_lens, const int* seq_of_row, int rows, int nh,
                              int kd, int vd, int max_blocks, int block_size, int num_rows, int window,
                              const float* sinks, float sm_scale, int dtype, void* stream) {
  if (rows <= 0 || nh <= 0) return 0;
  if (kd <= 0 || vd <= 0 || vd > kd || vd > 1024 || kd > 2048 || block_size <= 0 || max_blocks <= 0 || num_rows <= 0)
    return -10;
  RowsParams p = {};
  p.q_cat = q_cat; p.cache = cache; p.out = out; p.out_head_stride = out_head_stride; p.out_row_stride = out_row_stride;
  p.block_tables = block_tables; p.row_lens = row_lens; p.seq_of_row = seq_of_row; p.rows = rows;
  p.nh = nh; p.kd = kd; p.vd = vd; p.max_blocks = max_blocks; p.block_size = block_size; p.num_rows = num_rows;
  p.window = window; p.sm_scale = sm_scale; p.nkv = 1; p.x.maps = 1; p.x.sinks = sinks;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define FI_CALL(TT) return launch_rows<TT>(p, s)
  FI_BY_TYPE(dtype, FI_CALL)
#undef FI_CALL
  return 0;
}

// The same over separate key and value caches [blocks, nkv, block_size, kd | vd] (query head h reads key / value head
// h / (nh / nkv)): q [rows, nh, kd], out [rows, nh * vd]; row r sees the first row_lens[r] tokens (the last `window` of
// them) of sequence seq_of_row[r] (null: sequence r).  extra: see attn_extra.h, or null.  Two maps per head: q [rows, nh,
// kd / 2] with query heads 2 j and 2 j + 1 for output head j, key rows [map 1 | map 2], out [rows, nh / 2 * vd].
extern "C" int fi_attn_rows(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_tables,
                            const int* row_lens, const int* seq_of_row, int rows, int nh, int nkv, int kd, int vd,
                            int max_blocks, int block_size, int num_blocks, int window, const FiAttnExtra* extra,
                            float sm_scale, int dtype, void* stream) {
  if (rows <= 0 || nh <= 0) return 0;
  if (kd <= 0 || vd <= 0 || vd > 1024 || kd > 2048 || block_size <= 0 || max_blocks <= 0 || num_blocks <= 0 || nkv <= 0 ||
      nh % nkv != 0 || v_cache == nullptr)
    return -10;
  RowsParams p = {};
  if (!fi::take_extra(p, extra, vd, nh, nkv) || p.x.out_dim != vd || kd % p.x.maps != 0) return -10;
  p.q_cat = q; p.cache = k_cache; p.v_cache = v_cache; p.out = out; p.out_head_stride = vd;
  p.out_row_stride = static_cast<long>(nh / p.x.maps) * vd; p.block_tables = block_tables; p.row_lens = row_lens;
  p.seq_of_row = seq_of_row; p.rows = rows; p.nh = nh; p.nkv = nkv; p.kd = kd; p.vd = vd;
  p.max_blocks = max_blocks; p.block_size = block_size; p.num_rows = num_blocks * block_size; p.window = window;
  p.sm_scale = sm_scale;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define FI_CALL(TT) return launch_rows<TT>(p, s)
  FI_BY_TYPE(dtype, FI_CALL)
#undef FI_CALL
  return 0;
}
