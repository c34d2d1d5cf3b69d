// Residual stream of decoders whose sublayers read a short causal convolution of the normalised stream, and mixers that
// read several blends of the present and the previous input.  With x^ = x / rms(x) (32-bit), a layer's inputs are
//
//   h1_t = sum_j a1_j x^_(t - taps + 1 + j)        h2_t = sum_j a2_j x^_(t - taps + 1 + j)          (per channel)
//   b^i_t = h1_t + (h1_(t-1) - h1_t) mu^i                                                         (blends, i < 5)
//
// where the caller folds the norm's weight w and the direct path into the taps, a_j = w (conv_j + [j = taps - 1]), so
// both sublayers share one x^ and one ring of its last taps + 1 values per request slot (position p in row p % (taps + 1);
// x^ is zero before the start of a sequence).
//
//   shift_rows_kernel   per token: the stream after a layer,
//                         start   v = norm(table[token] + pairs[row of (previous token, token)]) * w
//                         sum     v = x + y + f
//                         pair    v = x + norm(y) w_y + norm(y2) w_y2 + f      (f: dense feed-forward and / or chosen experts)
//                       and, from it, 1 / rms(v) (portions), norm(v) * w of chosen rows (the end of the model), or
//                       everything the next layer reads (one token per sequence: convolution from the ring)
//   shift_conv_kernel   portions: h1, h2 and the blends; a thread owns channels and slides along a tile of tokens
//
// A portion's ring is read and written by the tile that starts it, and by the same thread for a channel, so blocks never
// race; the remembered token is written one kernel after it was read.
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../common/launch.cuh"

namespace {

enum Mode : int { kStart = 0, kSum = 1, kPair = 2 };
enum Out : int { kInv = 0, kNorm = 1, kToken = 2 };
enum DType : int { kBf16 = 0, kFp16 = 1, kFp32 = 2 };
constexpr int kBlends = 5;

struct ShiftParams {
  int mode, out_kind, h_type;
  // start
  const long long* ids;      // [T]
  const void* table;         // [vocab, W] (h_type)
  const void* pairs;         // [buckets + 1, W] (h_type)
  long long mul_prev, mul_cur;
  int vocab, buckets;
  int* last_token;           // [slots]
  // sum, pair
  const float* x;            // [T, W]
  const void* y;             // [T, ldy] (h_type)
  const void* y2;            // [T, ldy2]
  const float* w_y;          // [W] (start: the weight of its norm)
  const float* w_y2;
  const void* f;             // [T, ldf] or null
  const void* routed;        // expert rows of pitch ldr, or null
  const int* slot_of;        // [T, top]; null: row = token * top + choice
  const float* route_w;      // [T, top]; null: route_c for every choice
  float route_c;
  float* x_out;              // [T, W] or null
  long ldy, ldy2, ldf, ldr;
  int top;
  // results
  float* inv;                // [T]
  const float* w_pre;        // kNorm: [W]
  const long long* sel;      // kNorm: token of each row, or null
  const float* a1;           // [taps, W]
  const float* a2;           // [taps, W] or null
  const float* mu;           // [5, W] or null
  float* ring;               // [slots, taps + 1, W]
  void* out;                 // [1 + (a2) + 5 (mu)] matrices [*, ldo], out_stride apart (h_type); kNorm: one
  long ldo, out_stride;
  const int* slots;          // [B]
  const int* seq_lens;       // [B] length after this step
  const int* cu_q;           // [B + 1] (portions)
  const int* tile_base;      // [B + 1] tiles before each sequence (shift_conv)
  int B, rows, W, taps, tile, num_slots;
  float eps;
};

template <int VEC, bool H16>
__device__ __forceinline__ void load_h(const void* p, long i, int type, float* v) {
  if constexpr (!H16) {
    if constexpr (VEC == 4) {
      const float4 f = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
      v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else {
      v[0] = reinterpret_cast<const float*>(p)[i];
    }
    return;
  }
  alignas(8) uint16_t raw[VEC];
  if constexpr (VEC == 4) *reinterpret_cast<uint2*>(raw) = *reinterpret_cast<const uint2*>(reinterpret_cast<const uint16_t*>(p) + i);
  else raw[0] = reinterpret_cast<const uint16_t*>(p)[i];
#pragma unroll
  for (int e = 0; e < VEC; ++e)
    v[e] = type == kBf16 ? __uint_as_float(static_cast<uint32_t>(raw[e]) << 16) : __half2float(__ushort_as_half(raw[e]));
}
template <int VEC>
__device__ __forceinline__ void load_f(const float* p, long i, float* v) { load_h<VEC, false>(p, i, kFp32, v); }

template <int VEC, bool H16>
__device__ __forceinline__ void store_h(void* p, long i, int type, const float* v) {
  if constexpr (!H16) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + i) = make_float4(v[0], v[1], v[2], v[3]);
    else reinterpret_cast<float*>(p)[i] = v[0];
    return;
  }
  alignas(8) uint16_t raw[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e)
    raw[e] = type == kBf16 ? __bfloat16_as_ushort(__float2bfloat16_rn(v[e])) : __half_as_ushort(__float2half_rn(v[e]));
  if constexpr (VEC == 4) *reinterpret_cast<uint2*>(reinterpret_cast<uint16_t*>(p) + i) = *reinterpret_cast<const uint2*>(raw);
  else reinterpret_cast<uint16_t*>(p)[i] = raw[0];
}

// Sums of two values over the TPR threads that share a row.
template <int TPR>
__device__ __forceinline__ void row_sums(float& a, float& b, float (*red)[16]) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    a += __shfl_xor_sync(0xffffffffu, a, o);
    b += __shfl_xor_sync(0xffffffffu, b, o);
  }
  if constexpr (TPR > 32) {
    __syncthreads();
    if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = a; red[1][threadIdx.x >> 5] = b; }
    __syncthreads();
    a = b = 0.f;
#pragma unroll
    for (int w = 0; w < TPR / 32; ++w) { a += red[0][w]; b += red[1][w]; }
  }
}

// The sequence a position of a running count belongs to.
__device__ __forceinline__ int find_seq(const int* base, int B, int at) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (base[mid] <= at) lo = mid; else hi = mid - 1;
  }
  return lo;
}

constexpr int block_threads(int tpr) { return tpr > 256 ? tpr : 256; }

// TOKEN: one token per sequence, what the next layer reads included; otherwise rows of portions or of the end of the model.
template <int TPR, int VEC, int NV, bool H16, bool TOKEN>
__global__ void __launch_bounds__(block_threads(TPR)) shift_rows_kernel(const ShiftParams p) {
  fi::pdl_launch_dependents();
  if constexpr (TOKEN) {                   // weights of a decode step come from memory: ask for them while the predecessor ends
    for (int c = static_cast<int>(threadIdx.x) % TPR * VEC; c < p.W; c += TPR * VEC) {
      if (p.w_y != nullptr) fi::prefetch_l2(p.w_y + c);
      if (p.w_y2 != nullptr) fi::prefetch_l2(p.w_y2 + c);
      for (int j = 0; j < p.taps; ++j) {
        fi::prefetch_l2(p.a1 + static_cast<long>(j) * p.W + c);
        if (p.a2 != nullptr) fi::prefetch_l2(p.a2 + static_cast<long>(j) * p.W + c);
      }
      if (p.mu != nullptr)
        for (int k = 0; k < kBlends; ++k) fi::prefetch_l2(p.mu + static_cast<long>(k) * p.W + c);
    }
  }
  fi::pdl_wait();
  __shared__ float red[2][16];
  constexpr int kRowsPerBlock = block_threads(TPR) / TPR, N = NV * VEC;
  const int r = blockIdx.x * kRowsPerBlock + (kRowsPerBlock == 1 ? 0 : static_cast<int>(threadIdx.x) / TPR);
  const int tid = kRowsPerBlock == 1 ? threadIdx.x : threadIdx.x % TPR;
  if (r >= p.rows) return;                 // uniform over the threads of a row
  const long t = p.sel != nullptr ? static_cast<long>(p.sel[r]) : r;
  const int W = p.W;
  const float inv_n = 1.f / static_cast<float>(W);
  int len = 0, slot = 0;
  const int n_out = 1 + (p.a2 != nullptr) + (p.mu != nullptr ? kBlends : 0);
  if constexpr (TOKEN) {
    len = p.seq_lens[r];
    slot = p.slots[r];
    if (len <= 0 || slot < 0 || slot >= p.num_slots) {       // padded row of a decode bucket
      float zero[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) zero[e] = 0.f;
      for (int c = tid * VEC; c < W; c += TPR * VEC) {
        if (p.x_out != nullptr) store_h<VEC, false>(p.x_out, t * W + c, kFp32, zero);
        for (int i = 0; i < n_out; ++i) store_h<VEC, H16>(p.out, i * p.out_stride + r * p.ldo + c, p.h_type, zero);
      }
      return;
    }
  }

  // everything that is read is requested ahead of the first reduction
  float v[N], y[N], z[N];
  if (p.mode == kStart) {
    long long id = p.ids[t], prev = -1;
    if constexpr (TOKEN) {
      if (len > 1) prev = p.last_token[slot];
    } else {
      const int b = find_seq(p.cu_q, p.B, static_cast<int>(t));
      const int idx = static_cast<int>(t) - p.cu_q[b], n = p.cu_q[b + 1] - p.cu_q[b], s = p.slots[b];
      if (idx > 0) prev = p.ids[t - 1];
      else if (p.seq_lens[b] > n && s >= 0 && s < p.num_slots) prev = p.last_token[s];
    }
    const long long now = id;
    if (id < 0 || id >= p.vocab) id = 0;
    long long pr = p.buckets;
    if (prev >= 0) {
      pr = (prev * p.mul_prev + now * p.mul_cur) % p.buckets;
      if (pr < 0) pr += p.buckets;
    }
    float ss = 0.f, none = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[i * VEC + e] = y[i * VEC + e] = 0.f;
      if (c < W) {
        load_h<VEC, H16>(p.table, id * W + c, p.h_type, v + i * VEC);
        load_h<VEC, H16>(p.pairs, pr * W + c, p.h_type, y + i * VEC);
      }
    }
#pragma unroll
    for (int i = 0; i < N; ++i) { v[i] += y[i]; ss = fmaf(v[i], v[i], ss); }
    row_sums<TPR>(ss, none, red);
    if constexpr (TOKEN) {
      __syncwarp();
      if (tid == 0) p.last_token[slot] = static_cast<int>(now);     // every thread of the row has read it
    }
    const float inv = 1.f / sqrtf(ss * inv_n + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c < W) {
        float w[VEC];
        load_f<VEC>(p.w_y, c, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[i * VEC + e] *= inv * w[e];
      }
    }
  } else {
    const bool pair = p.mode == kPair;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[i * VEC + e] = y[i * VEC + e] = z[i * VEC + e] = 0.f;
      if (c < W) {
        load_f<VEC>(p.x, t * W + c, v + i * VEC);
        load_h<VEC, H16>(p.y, t * p.ldy + c, p.h_type, y + i * VEC);
        if (pair) load_h<VEC, H16>(p.y2, t * p.ldy2 + c, p.h_type, z + i * VEC);
      }
    }
    if (p.f != nullptr) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * TPR + tid) * VEC;
        if (c < W) {
          float g[VEC];
          load_h<VEC, H16>(p.f, t * p.ldf + c, p.h_type, g);
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[i * VEC + e] += g[e];
        }
      }
    }
    if (p.routed != nullptr) {
#pragma unroll 4
      for (int k = 0; k < p.top; ++k) {
        const long at = t * p.top + k;
        const long s = p.slot_of != nullptr ? p.slot_of[at] : at;
        const float w = s < 0 ? 0.f : p.route_w != nullptr ? p.route_w[at] : p.route_c;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = (i * TPR + tid) * VEC;
          if (c < W && s >= 0) {
            float q[VEC];
            load_h<VEC, H16>(p.routed, s * p.ldr + c, p.h_type, q);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[i * VEC + e] = fmaf(w, q[e], v[i * VEC + e]);
          }
        }
      }
    }
    if (pair) {
      float sy = 0.f, sz = 0.f;
#pragma unroll
      for (int i = 0; i < N; ++i) { sy = fmaf(y[i], y[i], sy); sz = fmaf(z[i], z[i], sz); }
      row_sums<TPR>(sy, sz, red);
      const float iy = 1.f / sqrtf(sy * inv_n + p.eps), iz = 1.f / sqrtf(sz * inv_n + p.eps);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * TPR + tid) * VEC;
        if (c < W) {
          float wy[VEC], wz[VEC];
          load_f<VEC>(p.w_y, c, wy);
          load_f<VEC>(p.w_y2, c, wz);
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[i * VEC + e] += fmaf(y[i * VEC + e] * iy, wy[e], z[i * VEC + e] * iz * wz[e]);
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < N; ++i) v[i] += y[i];
    }
  }

  // what the ring contributes does not wait for this token's norm: partial h1 and h2, and the previous token's h1
  [[maybe_unused]] float s1[TOKEN ? N : 1], s2[TOKEN ? N : 1], before[TOKEN ? N : 1];
  [[maybe_unused]] const int pos = len - 1, R = p.taps + 1;
  [[maybe_unused]] float* ring = TOKEN ? p.ring + static_cast<long>(slot) * R * W : nullptr;
  if constexpr (TOKEN) {
#pragma unroll
    for (int i = 0; i < N; ++i) s1[i] = s2[i] = before[i] = 0.f;
    auto back = [&](int j) {               // j tokens back
      if (j > p.taps || pos - j < 0) return;
      const float* row = ring + static_cast<long>((pos - j) % R) * W;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * TPR + tid) * VEC;
        if (c < W) {
          float u[VEC], a[VEC];
          load_f<VEC>(row, c, u);
          if (p.mu != nullptr) {
            load_f<VEC>(p.a1, static_cast<long>(p.taps - j) * W + c, a);
#pragma unroll
            for (int e = 0; e < VEC; ++e) before[i * VEC + e] = fmaf(a[e], u[e], before[i * VEC + e]);
          }
          if (j < p.taps) {
            load_f<VEC>(p.a1, static_cast<long>(p.taps - 1 - j) * W + c, a);
#pragma unroll
            for (int e = 0; e < VEC; ++e) s1[i * VEC + e] = fmaf(a[e], u[e], s1[i * VEC + e]);
            if (p.a2 != nullptr) {
              load_f<VEC>(p.a2, static_cast<long>(p.taps - 1 - j) * W + c, a);
#pragma unroll
              for (int e = 0; e < VEC; ++e) s2[i * VEC + e] = fmaf(a[e], u[e], s2[i * VEC + e]);
            }
          }
        }
      }
    };
#pragma unroll
    for (int j = 1; j <= 4; ++j) back(j);
    for (int j = 5; j <= p.taps; ++j) back(j);
  }

  float ss = 0.f, none = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * TPR + tid) * VEC;
    if (c < W) {
      if (p.x_out != nullptr) store_h<VEC, false>(p.x_out, t * W + c, kFp32, v + i * VEC);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(v[i * VEC + e], v[i * VEC + e], ss);
    }
  }
  row_sums<TPR>(ss, none, red);
  const float inv = 1.f / sqrtf(ss * inv_n + p.eps);
  if constexpr (!TOKEN) {
    if (p.out_kind == kInv) {
      if (tid == 0) p.inv[t] = inv;
      return;
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c < W) {
        float w[VEC];
        load_f<VEC>(p.w_pre, c, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) w[e] *= v[i * VEC + e] * inv;
        store_h<VEC, H16>(p.out, r * p.ldo + c, p.h_type, w);
      }
    }
  } else {
    float* mine = ring + static_cast<long>(pos % R) * W;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c >= W) continue;
      float a[VEC], h[VEC], n[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) n[e] = v[i * VEC + e] * inv;
      store_h<VEC, false>(mine, c, kFp32, n);
      load_f<VEC>(p.a1, static_cast<long>(p.taps - 1) * W + c, a);
#pragma unroll
      for (int e = 0; e < VEC; ++e) h[e] = fmaf(a[e], n[e], s1[i * VEC + e]);
      long at = static_cast<long>(r) * p.ldo + c;
      store_h<VEC, H16>(p.out, at, p.h_type, h);
      if (p.a2 != nullptr) {
        float g[VEC];
        load_f<VEC>(p.a2, static_cast<long>(p.taps - 1) * W + c, a);
#pragma unroll
        for (int e = 0; e < VEC; ++e) g[e] = fmaf(a[e], n[e], s2[i * VEC + e]);
        at += p.out_stride;
        store_h<VEC, H16>(p.out, at, p.h_type, g);
      }
      if (p.mu != nullptr) {
#pragma unroll
        for (int k = 0; k < kBlends; ++k) {
          float m[VEC];
          load_f<VEC>(p.mu, static_cast<long>(k) * W + c, m);
#pragma unroll
          for (int e = 0; e < VEC; ++e) m[e] = fmaf(before[i * VEC + e] - h[e], m[e], h[e]);
          at += p.out_stride;
          store_h<VEC, H16>(p.out, at, p.h_type, m);
        }
      }
    }
  }
}

// Stores in a type known at compile time (the convolution is bound by its instructions).
template <int VEC, int H>
__device__ __forceinline__ void store_as(void* p, long i, const float* v) {
  if constexpr (H == kFp32) {
    store_h<VEC, false>(p, i, kFp32, v);
  } else if constexpr (VEC == 4 && H == kBf16) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(reinterpret_cast<uint16_t*>(p) + i) =
        make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
    store_h<VEC, true>(p, i, H, v);
  }
}

// KT >= taps: registers of the sliding window (leading taps of weight zero).  MU: blends are formed.
template <int KT, int VEC, int H, bool MU>
__global__ void __launch_bounds__(128, KT > 4 ? 1 : MU ? 4 : 6) shift_conv_kernel(const ShiftParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  const int W = p.W, taps = p.taps, R = taps + 1;
  const int b = find_seq(p.tile_base, p.B, blockIdx.x);
  const int i0 = (static_cast<int>(blockIdx.x) - p.tile_base[b]) * p.tile;
  const int t_begin = p.cu_q[b], n = p.cu_q[b + 1] - t_begin;
  if (i0 < 0 || i0 >= n) return;
  const int pos0 = p.seq_lens[b] - n, slot = p.slots[b];
  if (slot < 0 || slot >= p.num_slots) return;
  if (i0 == 0 && blockIdx.y == 0 && threadIdx.x == 0 && p.last_token != nullptr)
    p.last_token[slot] = static_cast<int>(p.ids[t_begin + n - 1]);
  const int c = (blockIdx.y * 128 + threadIdx.x) * VEC;
  if (c >= W) return;
  float* ring = p.ring + static_cast<long>(slot) * R * W + c;
  auto unit = [&](int i, float* v) {       // x^ of the portion's token i
    load_f<VEC>(p.x, static_cast<long>(t_begin + i) * W + c, v);
    const float inv = p.inv[t_begin + i];
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] *= inv;
  };
  const float* second = p.a2 != nullptr ? p.a2 : p.a1;
  constexpr int HIST = MU ? KT : KT - 1;   // tokens before the present four; the blends also need the convolution one token back
  float a1[KT][VEC], a2[KT][VEC], mu[MU ? kBlends : 1][VEC], seq[HIST + 4][VEC], prev[VEC];
#pragma unroll
  for (int j = 0; j < KT; ++j) {
    const int tap = j - (KT - taps);
    load_f<VEC>(p.a1, static_cast<long>(max(tap, 0)) * W + c, a1[j]);
    load_f<VEC>(second, static_cast<long>(max(tap, 0)) * W + c, a2[j]);
    if (tap < 0)
#pragma unroll
      for (int e = 0; e < VEC; ++e) a1[j][e] = a2[j][e] = 0.f;
  }
  // loads take no branches, so that they are in flight together
  if (i0 > 0) {                            // a tile holds at least taps tokens
#pragma unroll
    for (int j = 0; j < HIST; ++j) unit(max(i0 - HIST + j, 0), seq[j]);
  } else {
#pragma unroll
    for (int j = 0; j < HIST; ++j) {
      const int i = j - HIST;
#pragma unroll
      for (int e = 0; e < VEC; ++e) seq[j][e] = 0.f;
      if (-i <= taps && pos0 + i >= 0) load_f<VEC>(ring, static_cast<long>((pos0 + i) % R) * W, seq[j]);
    }
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) prev[e] = 0.f;
  if constexpr (MU) {
#pragma unroll
    for (int k = 0; k < kBlends; ++k) load_f<VEC>(p.mu, static_cast<long>(k) * W + c, mu[k]);
#pragma unroll
    for (int j = 0; j < KT; ++j)
#pragma unroll
      for (int e = 0; e < VEC; ++e) prev[e] = fmaf(a1[j][e], seq[j][e], prev[e]);
  }
  const int i_end = min(n, i0 + p.tile);
  for (int i = i0; i < i_end; i += 4) {
#pragma unroll
    for (int u = 0; u < 4; ++u) unit(min(i + u, i_end - 1), seq[HIST + u]);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (i + u >= i_end) break;
      constexpr int kFirst = HIST - KT + 1;                  // seq[kFirst + u + KT - 1] is token i + u
      float h[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) h[e] = 0.f;
#pragma unroll
      for (int j = 0; j < KT; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) h[e] = fmaf(a1[j][e], seq[kFirst + u + j][e], h[e]);
      long at = static_cast<long>(t_begin + i + u) * p.ldo + c;
      store_as<VEC, H>(p.out, at, h);
      if (p.a2 != nullptr) {
        float g[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) g[e] = 0.f;
#pragma unroll
        for (int j = 0; j < KT; ++j)
#pragma unroll
          for (int e = 0; e < VEC; ++e) g[e] = fmaf(a2[j][e], seq[kFirst + u + j][e], g[e]);
        at += p.out_stride;
        store_as<VEC, H>(p.out, at, g);
      }
      if constexpr (MU) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) prev[e] -= h[e];
#pragma unroll
        for (int k = 0; k < kBlends; ++k) {
          float m[VEC];
#pragma unroll
          for (int e = 0; e < VEC; ++e) m[e] = fmaf(prev[e], mu[k][e], h[e]);
          at += p.out_stride;
          store_as<VEC, H>(p.out, at, m);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) prev[e] = h[e];
      }
    }
#pragma unroll
    for (int j = 0; j < HIST; ++j)
#pragma unroll
      for (int e = 0; e < VEC; ++e) seq[j][e] = seq[j + 4][e];
  }
  if (i0 == 0)                              // what the next step of this sequence looks back at
    for (int i = max(0, n - taps); i < n; ++i) {
      float x[VEC];
      unit(i, x);
      store_h<VEC, false>(ring, static_cast<long>((pos0 + i) % R) * W, kFp32, x);
    }
}

template <int TPR, int VEC, int NV>
int launch_rows(const ShiftParams& p, cudaStream_t s) {
  constexpr int threads = block_threads(TPR), per = threads / TPR;
  const dim3 g(static_cast<unsigned>((p.rows + per - 1) / per));
  auto kern = p.out_kind == kToken ? (p.h_type == kFp32 ? shift_rows_kernel<TPR, VEC, NV, false, true> : shift_rows_kernel<TPR, VEC, NV, true, true>)
                                   : (p.h_type == kFp32 ? shift_rows_kernel<TPR, VEC, NV, false, false> : shift_rows_kernel<TPR, VEC, NV, true, false>);
  return static_cast<int>(fi::launch_kernel(kern, g, dim3(threads), 0, s, 0, p));
}

template <int KT, int VEC>
int launch_conv(const ShiftParams& p, int tiles, cudaStream_t s) {
  const dim3 g(tiles, (p.W + 128 * VEC - 1) / (128 * VEC));
  auto kern = p.h_type == kBf16   ? (p.mu != nullptr ? shift_conv_kernel<KT, VEC, kBf16, true> : shift_conv_kernel<KT, VEC, kBf16, false>)
              : p.h_type == kFp16 ? (p.mu != nullptr ? shift_conv_kernel<KT, VEC, kFp16, true> : shift_conv_kernel<KT, VEC, kFp16, false>)
                                  : (p.mu != nullptr ? shift_conv_kernel<KT, VEC, kFp32, true> : shift_conv_kernel<KT, VEC, kFp32, false>);
  return static_cast<int>(fi::launch_kernel(kern, g, dim3(128), 0, s, 0, p));
}

bool aligned(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

int dispatch_rows(const ShiftParams& p, cudaStream_t s) {
  const bool vec4 = p.W % 4 == 0 && (p.ldy | p.ldy2 | p.ldf | p.ldr | p.ldo | p.out_stride) % 4 == 0 && aligned(p.table) && aligned(p.pairs) &&
                    aligned(p.x) && aligned(p.y) && aligned(p.y2) && aligned(p.w_y) && aligned(p.w_y2) && aligned(p.f) &&
                    aligned(p.routed) && aligned(p.x_out) && aligned(p.w_pre) && aligned(p.a1) && aligned(p.a2) && aligned(p.mu) &&
                    aligned(p.ring) && aligned(p.out);
  const int W = p.W;
  if (!vec4) {
    if (W <= 32) return launch_rows<32, 1, 1>(p, s);
    if (W <= 1024) return launch_rows<256, 1, 4>(p, s);
    if (W <= 4096) return launch_rows<256, 1, 16>(p, s);
    return -11;
  }
  const bool few = p.rows < 2048;          // too few warps to fill the device
  if (W <= 128) return launch_rows<32, 4, 1>(p, s);
  if (!few || W <= 256) {
    if (W <= 256) return launch_rows<32, 4, 2>(p, s);
    if (W <= 512) return launch_rows<32, 4, 4>(p, s);
  }
  if (W <= 1024) return launch_rows<256, 4, 1>(p, s);
  if (W <= 2048) return few ? launch_rows<512, 4, 1>(p, s) : launch_rows<256, 4, 2>(p, s);
  if (W <= 4096) return launch_rows<512, 4, 2>(p, s);
  if (W <= 8192) return launch_rows<512, 4, 4>(p, s);
  return -11;
}

}  // namespace

// One layer boundary (or the start of the model) for rows of W channels.  src_mode: 0 start, 1 sum, 2 pair; out_kind: 0 writes
// inv [T] (and x_out), 1 writes norm(v) * w_pre of the rows sel (null: all), 2 one token per sequence: writes the next
// layer's inputs.  h_type (0 bf16, 1 fp16, 2 fp32): table, pairs, y, y2, f, routed and out.  Pointers that a mode does not
// use may be null.  x_out must not be x's tokens of another row (in place is fine).  Token ids outside the table read row 0.
extern "C" int fi_shift_rows(int src_mode, int out_kind, const long long* ids, const void* table, int vocab, const void* pairs,
                             int buckets, long mul_prev, long mul_cur, int* last_token, const float* x, const void* y,
                             long ldy, const void* y2, long ldy2, const float* w_y, const float* w_y2, const void* f, long ldf,
                             const void* routed, long ldr, const int* slot_of, const float* route_w, float route_c, int top, float* x_out,
                             float* inv, const float* w_pre, const long long* sel, const float* a1, const float* a2,
                             const float* mu, int taps, float* ring, void* out, long ldo, long out_stride, const int* slots,
                             const int* seq_lens, const int* cu_q, int B, int num_slots, int rows, int W, float eps, int h_type,
                             void* stream) {
  if (rows <= 0) return 0;
  if (W <= 0 || h_type < 0 || h_type > 2 || src_mode < 0 || src_mode > 2 || out_kind < 0 || out_kind > 2) return -10;
  if (src_mode == kStart && (ids == nullptr || table == nullptr || pairs == nullptr || last_token == nullptr || w_y == nullptr ||
                             vocab <= 0 || buckets <= 0 || slots == nullptr || seq_lens == nullptr))
    return -10;
  if (src_mode != kStart && (x == nullptr || y == nullptr)) return -10;
  if (src_mode == kPair && (y2 == nullptr || w_y == nullptr || w_y2 == nullptr)) return -10;
  if (routed != nullptr && top <= 0) return -10;
  if (out_kind == kInv && inv == nullptr) return -10;
  if (out_kind == kNorm && (w_pre == nullptr || out == nullptr)) return -10;
  if (out_kind == kToken && (a1 == nullptr || ring == nullptr || out == nullptr || slots == nullptr || seq_lens == nullptr || taps <= 0))
    return -10;
  if (out_kind != kToken && src_mode == kStart && (cu_q == nullptr || B <= 0)) return -10;
  ShiftParams p = {};
  p.mode = src_mode; p.out_kind = out_kind; p.h_type = h_type; p.ids = ids; p.table = table; p.vocab = vocab; p.pairs = pairs;
  p.buckets = buckets; p.mul_prev = mul_prev; p.mul_cur = mul_cur; p.last_token = last_token; p.x = x; p.y = y; p.ldy = ldy;
  p.y2 = y2; p.ldy2 = ldy2; p.w_y = w_y; p.w_y2 = w_y2; p.f = f; p.ldf = ldf; p.routed = routed; p.ldr = ldr;
  p.slot_of = slot_of; p.route_w = route_w; p.route_c = route_c; p.top = top; p.x_out = x_out; p.inv = inv; p.w_pre = w_pre; p.sel = sel; p.a1 = a1;
  p.a2 = a2; p.mu = mu; p.taps = taps; p.ring = ring; p.out = out; p.ldo = ldo; p.out_stride = out_stride; p.slots = slots;
  p.seq_lens = seq_lens; p.cu_q = cu_q; p.B = B; p.num_slots = num_slots; p.rows = rows; p.W = W; p.eps = eps;
  return dispatch_rows(p, reinterpret_cast<cudaStream_t>(stream));
}

// Inputs of a layer for portions of sequences: x fp32 [T, W] with inv [T]; tile_base int32 [B + 1] counts tiles of `tile`
// tokens (at least taps), n_tiles its last entry; ids and last_token (both or neither): remembers each portion's last token.
extern "C" int fi_shift_conv(const float* x, const float* inv, const float* a1, const float* a2, const float* mu, int taps,
                             float* ring, void* out, long ldo, long out_stride, const long long* ids, int* last_token,
                             const int* slots, const int* seq_lens, const int* cu_q, const int* tile_base, int n_tiles, int tile,
                             int B, int num_slots, int W, int h_type, void* stream) {
  if (n_tiles <= 0 || B <= 0) return 0;
  if (W <= 0 || taps <= 0 || taps > 16 || tile < taps || h_type < 0 || h_type > 2 || (ids == nullptr) != (last_token == nullptr)) return -10;
  ShiftParams p = {};
  p.x = x; p.inv = const_cast<float*>(inv); p.a1 = a1; p.a2 = a2; p.mu = mu; p.taps = taps; p.ring = ring; p.out = out; p.ldo = ldo;
  p.out_stride = out_stride; p.ids = ids; p.last_token = last_token; p.slots = slots; p.seq_lens = seq_lens; p.cu_q = cu_q;
  p.tile_base = tile_base; p.tile = tile; p.B = B; p.num_slots = num_slots; p.W = W; p.h_type = h_type;
  const bool vec4 = W % 4 == 0 && (ldo | out_stride) % 4 == 0 && aligned(x) && aligned(a1) && aligned(a2) && aligned(mu) &&
                    aligned(ring) && aligned(out);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (taps <= 4) return vec4 ? launch_conv<4, 4>(p, n_tiles, s) : launch_conv<4, 1>(p, n_tiles, s);
  if (taps <= 8) return vec4 ? launch_conv<8, 4>(p, n_tiles, s) : launch_conv<8, 1>(p, n_tiles, s);
  return launch_conv<16, 1>(p, n_tiles, s);
}
