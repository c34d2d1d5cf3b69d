// Residual-stream kernels: decoders whose sublayers are normalised on both sides and whose layers read a weighted
// average of everything before them, decoders whose sublayers read one norm side by side, and decoders that normalise
// only what a sublayer returns.  The stream and every norm are 32-bit; the sublayers' inputs and outputs may be 16-bit.
//
//   start    v = table[token] * scale                                  X_0 = v
//   add      v = x + y + sum_k w_k e_(slot k)                          x   = v     (y: mixer, e: routed experts' rows)
//   step     v = x + norm(y) * w_post                                  x   = v
//   post     v = x + norm(y + sum_k w_k e_k) * w_post                  x   = v     (e_k: routed experts' rows, or x)
//   average  X_n = x + norm(y) * w_post;  v = sum_{j<=n} a_j X_j        x   = v
//   each:    h = norm(v) * w_pre          (what the next sublayer reads; start, post: v itself without w_pre)
//
// The norm is an RMS norm over equal consecutive parts ("groups") of the vector, so a group of one token needs
// nothing from any other group: the unit of work is a (token, group) row.  Steps with many tokens give a row to a
// warp, steps with few tokens (decode) and long rows to a block, whose threads then fetch the whole history at once.
// Rows keep their values in registers between the two norms: one read of y and x, one write of x and h.
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../common/launch.cuh"

namespace {

enum Mode : int { kStart = 0, kStep = 1, kAverage = 2, kAdd = 3, kPost = 4 };
enum DType : int { kBf16 = 0, kFp16 = 1, kFp32 = 2 };

struct StreamParams {
  const void* y;         // [*, ldy] sublayer output (type y_type); kPost: null = zeros
  const float* x;        // [*, W] stream before the sublayer
  const void* table;     // kStart: [V, W] embedding (type h_type)
  const long long* ids;  // kStart: token per row
  const float* w_post;   // [W]
  const float* w_pre;    // [W] or null (no h)
  float* hist;           // kAverage: [n, T, W] X_0 .. X_(n-1); slot n is written
  const float* avg;      // kAverage: [n + 1]
  float* x_out;          // [*, W] or null
  void* h;               // [*, ldh] (type h_type)
  const long long* sel;  // optional: output row r comes from token sel[r]; x_out is not written then
  const void* routed;    // kAdd, kPost: expert outputs (type y_type), rows of pitch ldr, or null
  const int* slot_of;    // kAdd, kPost: [*, top] row of each (token, choice), < 0: none; null: row = token * top + choice
  const float* route_w;  // kAdd, kPost: [*, top]
  long ldy, ldh, hist_stride, ldr;
  float scale;           // kStart
  int top, pass_through; // pass_through: a choice without a row stands for x itself (kPost)
  int rows, W, group, groups, n, y_type, h_type, vocab;
  float eps;
};

// 16-bit or 32-bit storage is a compile-time choice (H16): a branch around every load would keep the loads of a row
// from being issued together.  bf16 / fp16 is a select on the loaded bits.
template <int VEC, bool H16>
__device__ __forceinline__ void load_any(const void* p, long i, int type, float* v) {
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
  if constexpr (VEC == 4) {
    *reinterpret_cast<uint2*>(raw) = *reinterpret_cast<const uint2*>(reinterpret_cast<const uint16_t*>(p) + i);
  } else {
    raw[0] = reinterpret_cast<const uint16_t*>(p)[i];
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e)
    v[e] = type == kBf16 ? __uint_as_float(static_cast<uint32_t>(raw[e]) << 16)
                         : __half2float(__ushort_as_half(raw[e]));
}

template <int VEC, bool H16>
__device__ __forceinline__ void store_any(void* p, long i, int type, const float* v) {
  if constexpr (!H16) {
    if constexpr (VEC == 4)
      *reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + i) = make_float4(v[0], v[1], v[2], v[3]);
    else
      reinterpret_cast<float*>(p)[i] = v[0];
    return;
  }
  alignas(8) uint16_t raw[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e)
    raw[e] = type == kBf16 ? __bfloat16_as_ushort(__float2bfloat16_rn(v[e])) : __half_as_ushort(__float2half_rn(v[e]));
  if constexpr (VEC == 4)
    *reinterpret_cast<uint2*>(reinterpret_cast<uint16_t*>(p) + i) = *reinterpret_cast<const uint2*>(raw);
  else
    reinterpret_cast<uint16_t*>(p)[i] = raw[0];
}

// Sum over the TPR threads that share a row (a warp, or the whole block).
template <int TPR>
__device__ __forceinline__ float row_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if constexpr (TPR > 32) {
    __syncthreads();                       // the previous use of `red` is over
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    v = 0.f;
#pragma unroll
    for (int w = 0; w < TPR / 32; ++w) v += red[w];
  }
  return v;
}

// Threads of a block whose rows take tpr threads each.
constexpr int block_threads(int tpr) { return tpr > 256 ? tpr : 256; }

template <int MODE, int TPR, int VEC, int NV, bool H16>
__global__ void __launch_bounds__(block_threads(TPR)) stream_kernel(const StreamParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  __shared__ float red[16];
  constexpr int kRowsPerBlock = block_threads(TPR) / TPR;
  const int row = blockIdx.x * kRowsPerBlock + (kRowsPerBlock == 1 ? 0 : static_cast<int>(threadIdx.x) / TPR);
  const int tid = kRowsPerBlock == 1 ? threadIdx.x : threadIdx.x % TPR;
  if (row >= p.rows * p.groups) return;    // uniform over the threads of a row
  const int r = row / p.groups, g = row % p.groups;
  const long t = p.sel != nullptr ? static_cast<long>(p.sel[r]) : r;
  const int c0 = g * p.group;              // first channel of the group
  float v[NV * VEC];
  const float inv_n = 1.f / static_cast<float>(p.group);

  if constexpr (MODE == kStart) {
    long id = static_cast<long>(p.ids[t]);
    if (id < 0 || id >= p.vocab) id = 0;   // padded rows of a decode bucket carry stale ids
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c < p.group) load_any<VEC, H16>(p.table, id * p.W + c0 + c, p.h_type, v + i * VEC);
      else
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[i * VEC + e] = 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[i * VEC + e] *= p.scale;
    }
  } else if constexpr (MODE == kAdd) {
    float yv[NV * VEC];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c < p.group) {
        load_any<VEC, H16>(p.y, t * p.ldy + c0 + c, p.y_type, yv + i * VEC);
        load_any<VEC, false>(p.x, t * p.W + c0 + c, kFp32, v + i * VEC);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) { v[i * VEC + e] = 0.f; yv[i * VEC + e] = 0.f; }
      }
    }
    if (p.routed != nullptr) {
#pragma unroll 4
      for (int k = 0; k < p.top; ++k) {
        const long at = t * p.top + k;
        const long slot = p.slot_of != nullptr ? p.slot_of[at] : at;
        const float w = slot >= 0 ? p.route_w[at] : 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = (i * TPR + tid) * VEC;
          if (c < p.group && slot >= 0) {
            float e4[VEC];
            load_any<VEC, H16>(p.routed, slot * p.ldr + c0 + c, p.y_type, e4);
#pragma unroll
            for (int e = 0; e < VEC; ++e) yv[i * VEC + e] = fmaf(w, e4[e], yv[i * VEC + e]);
          }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NV * VEC; ++i) v[i] += yv[i];
  } else {
    float xv[NV * VEC];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c < p.group) {
        if (MODE != kPost || p.y != nullptr) {
          load_any<VEC, H16>(p.y, t * p.ldy + c0 + c, p.y_type, v + i * VEC);
        } else {
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[i * VEC + e] = 0.f;
        }
        load_any<VEC, false>(p.x, t * p.W + c0 + c, kFp32, xv + i * VEC);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) { v[i * VEC + e] = 0.f; xv[i * VEC + e] = 0.f; }
      }
    }
    if constexpr (MODE == kPost) {
      float through = 0.f;                 // weight of x itself
      if (p.routed != nullptr) {
#pragma unroll 4
        for (int k = 0; k < p.top; ++k) {
          const long at = t * p.top + k;
          const long slot = p.slot_of != nullptr ? p.slot_of[at] : at;
          const float w = p.route_w[at];
          if (slot < 0) through += w;
#pragma unroll
          for (int i = 0; i < NV; ++i) {
            const int c = (i * TPR + tid) * VEC;
            if (c < p.group && slot >= 0) {
              float e4[VEC];
              load_any<VEC, H16>(p.routed, slot * p.ldr + c0 + c, p.y_type, e4);
#pragma unroll
              for (int e = 0; e < VEC; ++e) v[i * VEC + e] = fmaf(w, e4[e], v[i * VEC + e]);
            }
          }
        }
      }
      if (p.pass_through) {
#pragma unroll
        for (int i = 0; i < NV * VEC; ++i) v[i] = fmaf(through, xv[i], v[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < NV * VEC; ++i) ss += v[i] * v[i];
    if constexpr (MODE == kPost) {         // the weight is applied ahead of the reduction: less to do behind it
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * TPR + tid) * VEC;
        if (c < p.group) {
          float w[VEC];
          load_any<VEC, false>(p.w_post, c0 + c, kFp32, w);
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[i * VEC + e] *= w[e];
        }
      }
    }
    const float inv = 1.f / sqrtf(row_sum<TPR>(ss, red) * inv_n + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c < p.group) {
        if constexpr (MODE == kPost) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[i * VEC + e] = fmaf(v[i * VEC + e], inv, xv[i * VEC + e]);
        } else {
          float w[VEC];
          load_any<VEC, false>(p.w_post, c0 + c, kFp32, w);
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[i * VEC + e] = fmaf(v[i * VEC + e] * inv, w[e], xv[i * VEC + e]);
        }
      }
    }
    if constexpr (MODE == kAverage) {
      const float an = p.avg[p.n];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = (i * TPR + tid) * VEC;
        if (c < p.group && p.sel == nullptr)
          store_any<VEC, false>(p.hist, p.n * p.hist_stride + t * p.W + c0 + c, kFp32, v + i * VEC);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[i * VEC + e] *= an;
      }
      const float* hrow = p.hist + t * p.W + c0;
#pragma unroll 4
      for (int j = 0; j < p.n; ++j) {
        const float a = p.avg[j];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = (i * TPR + tid) * VEC;
          if (c < p.group) {
            float o[VEC];
            load_any<VEC, false>(hrow + j * p.hist_stride, c, kFp32, o);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[i * VEC + e] = fmaf(a, o[e], v[i * VEC + e]);
          }
        }
      }
    }
  }

  if (p.x_out != nullptr) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c < p.group) store_any<VEC, false>(p.x_out, t * p.W + c0 + c, kFp32, v + i * VEC);
    }
  }
  if (p.w_pre != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c < p.group)
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss += v[i * VEC + e] * v[i * VEC + e];
    }
    const float inv = 1.f / sqrtf(row_sum<TPR>(ss, red) * inv_n + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c < p.group) {
        float w[VEC], o[VEC];
        load_any<VEC, false>(p.w_pre, c0 + c, kFp32, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) o[e] = v[i * VEC + e] * inv * w[e];
        store_any<VEC, H16>(p.h, static_cast<long>(r) * p.ldh + c0 + c, p.h_type, o);
      }
    }
  } else if ((MODE == kStart || MODE == kPost) && p.h != nullptr) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * VEC;
      if (c < p.group) store_any<VEC, H16>(p.h, static_cast<long>(r) * p.ldh + c0 + c, p.h_type, v + i * VEC);
    }
  }
}

template <int MODE, int TPR, int VEC, int NV>
int launch(const StreamParams& p, cudaStream_t s) {
  const long rows = static_cast<long>(p.rows) * p.groups;
  constexpr int threads = block_threads(TPR), per = threads / TPR;
  const long grid = (rows + per - 1) / per;
  if (grid > 2147483647l) return -10;
  const dim3 g(static_cast<unsigned>(grid));
  if (p.h_type == kFp32)
    return static_cast<int>(fi::launch_kernel(stream_kernel<MODE, TPR, VEC, NV, false>, g, dim3(threads), 0, s, 0, p));
  return static_cast<int>(fi::launch_kernel(stream_kernel<MODE, TPR, VEC, NV, true>, g, dim3(threads), 0, s, 0, p));
}

template <int MODE>
int dispatch(const StreamParams& p, bool vec4, cudaStream_t s) {
  const int g = p.group;
  if (!vec4) {
    if (g <= 32) return launch<MODE, 32, 1, 1>(p, s);
    if (g <= 1024) return launch<MODE, 256, 1, 4>(p, s);
    if (g <= 4096) return launch<MODE, 256, 1, 16>(p, s);
    return -11;
  }
  const bool few = static_cast<long>(p.rows) * p.groups < 2048;      // too few warps to fill the device
  if (g <= 128) return launch<MODE, 32, 4, 1>(p, s);
  if (!few || g <= 256) {
    if (g <= 256) return launch<MODE, 32, 4, 2>(p, s);
    if (g <= 512) return launch<MODE, 32, 4, 4>(p, s);
  }
  if (g <= 1024) return launch<MODE, 256, 4, 1>(p, s);
  if (g <= 2048) return launch<MODE, 256, 4, 2>(p, s);
  if constexpr (MODE == kPost) {      // everything it stores lies behind the reduction: more warps hide that
    if (g <= 4096) return launch<MODE, 512, 4, 2>(p, s);
    if (g <= 8192) return launch<MODE, 512, 4, 4>(p, s);
  } else {
    if (g <= 4096) return launch<MODE, 256, 4, 4>(p, s);
    if (g <= 8192) return launch<MODE, 256, 4, 8>(p, s);
  }
  return -11;
}

bool aligned(const void* p, unsigned a) { return (reinterpret_cast<uintptr_t>(p) & (a - 1)) == 0; }

}  // namespace

// X_0 = table[ids] * scale (32-bit) into x0, h = norm(X_0) * w_pre (w_pre null: h = X_0; h null: none).  h_type (0 bf16, 1 fp16, 2 fp32) is also the
// table's type.  Token ids outside the table read row 0.
extern "C" int fi_stream_start(const long long* ids, const void* table, int vocab, float scale, const float* w_pre,
                               float* x0, void* h, long ldh, int T, int W, int groups, float eps, int h_type,
                               void* stream) {
  if (T <= 0) return 0;
  if (W <= 0 || groups <= 0 || W % groups != 0 || h_type < 0 || h_type > 2 || vocab <= 0) return -10;
  StreamParams p = {};
  p.ids = ids; p.table = table; p.vocab = vocab; p.scale = scale; p.w_pre = w_pre; p.x_out = x0; p.h = h; p.ldh = ldh; p.rows = T; p.W = W;
  p.group = W / groups; p.groups = groups; p.eps = eps; p.h_type = h_type; p.y_type = h_type;
  const bool vec4 = p.group % 4 == 0 && ldh % 4 == 0 && aligned(table, 16) && aligned(x0, 16) && aligned(h, 16) &&
                    aligned(w_pre, 16);
  return dispatch<kStart>(p, vec4, reinterpret_cast<cudaStream_t>(stream));
}

// x_out = x + norm(y) * w_post; h = norm(x_out) * w_pre (w_pre null: no h).  x_out may be x.  y and h share a type.
extern "C" int fi_stream_step(const void* y, long ldy, int y_type, const float* x, const float* w_post,
                              const float* w_pre, float* x_out, void* h, long ldh, int h_type, int T, int W, int groups,
                              float eps, void* stream) {
  if (T <= 0) return 0;
  if (W <= 0 || groups <= 0 || W % groups != 0 || h_type < 0 || h_type > 2 || y_type != h_type) return -10;
  StreamParams p = {};
  p.y = y; p.ldy = ldy; p.y_type = y_type; p.x = x; p.w_post = w_post; p.w_pre = w_pre; p.x_out = x_out; p.h = h;
  p.ldh = ldh; p.h_type = h_type; p.rows = T; p.W = W; p.group = W / groups; p.groups = groups; p.eps = eps;
  const bool vec4 = p.group % 4 == 0 && ldh % 4 == 0 && ldy % 4 == 0 && aligned(y, 16) && aligned(x, 16) &&
                    aligned(x_out, 16) && aligned(h, 16) && aligned(w_post, 16) && aligned(w_pre, 16);
  return dispatch<kStep>(p, vec4, reinterpret_cast<cudaStream_t>(stream));
}

// X_n = x + norm(y) * w_post into slot n of hist [*, T, W] (slot pitch hist_stride elements), v = sum_j avg[j] X_j,
// x_out = v, h = norm(v) * w_pre.  sel (optional, int64 [rows]): only these tokens are wanted; row r of h belongs to
// token sel[r] and neither slot n nor x_out is written.
extern "C" int fi_stream_average(const void* y, long ldy, int y_type, const float* x, const float* w_post,
                                 const float* w_pre, float* hist, long hist_stride, const float* avg, int n,
                                 float* x_out, void* h, long ldh, int h_type, const long long* sel, int rows, int W,
                                 int groups, float eps, void* stream) {
  if (rows <= 0) return 0;
  if (W <= 0 || groups <= 0 || W % groups != 0 || h_type < 0 || h_type > 2 || y_type != h_type || n < 1) return -10;
  if (sel != nullptr && x_out != nullptr) return -10;
  StreamParams p = {};
  p.y = y; p.ldy = ldy; p.y_type = y_type; p.x = x; p.w_post = w_post; p.w_pre = w_pre; p.hist = hist;
  p.hist_stride = hist_stride; p.avg = avg; p.n = n; p.x_out = x_out; p.h = h; p.ldh = ldh; p.h_type = h_type;
  p.sel = sel; p.rows = rows; p.W = W; p.group = W / groups; p.groups = groups; p.eps = eps;
  const bool vec4 = p.group % 4 == 0 && ldh % 4 == 0 && ldy % 4 == 0 && hist_stride % 4 == 0 && aligned(y, 16) &&
                    aligned(x, 16) && aligned(x_out, 16) && aligned(h, 16) && aligned(hist, 16) && aligned(w_post, 16) &&
                    aligned(w_pre, 16);
  return dispatch<kAverage>(p, vec4, reinterpret_cast<cudaStream_t>(stream));
}

// v = x + y + sum_k route_w[t, k] routed[slot_of[t, k]]; x_out = v (may be x, or null), h = norm(v) * w_pre.  y, routed
// and h share a type.  routed null: no experts.  sel (optional, int64 [rows]): only these tokens are wanted; row r of h
// belongs to token sel[r] and x_out must be null.
extern "C" int fi_stream_add(const void* y, long ldy, int y_type, const float* x, const void* routed, long ldr,
                             const int* slot_of, const float* route_w, int top, const float* w_pre, float* x_out, void* h,
                             long ldh, int h_type, const long long* sel, int rows, int W, int groups, float eps,
                             void* stream) {
  if (rows <= 0) return 0;
  if (W <= 0 || groups <= 0 || W % groups != 0 || h_type < 0 || h_type > 2 || y_type != h_type || top < 0) return -10;
  if ((sel != nullptr && x_out != nullptr) || (routed != nullptr && (route_w == nullptr || top <= 0))) return -10;
  StreamParams p = {};
  p.y = y; p.ldy = ldy; p.y_type = y_type; p.x = x; p.routed = routed; p.ldr = ldr; p.slot_of = slot_of; p.route_w = route_w;
  p.top = top; p.w_pre = w_pre; p.x_out = x_out; p.h = h; p.ldh = ldh; p.h_type = h_type; p.sel = sel; p.rows = rows;
  p.W = W; p.group = W / groups; p.groups = groups; p.eps = eps;
  const bool vec4 = p.group % 4 == 0 && ldh % 4 == 0 && ldy % 4 == 0 && ldr % 4 == 0 && aligned(y, 16) && aligned(x, 16) &&
                    aligned(x_out, 16) && aligned(h, 16) && aligned(routed, 16) && aligned(w_pre, 16);
  return dispatch<kAdd>(p, vec4, reinterpret_cast<cudaStream_t>(stream));
}

// v = x + norm(y + sum_k route_w[t, k] routed[slot_of[t, k]]) * w_post; x_out = v (may be x, or null); h = norm(v) *
// w_pre, or v itself without w_pre (h null: none).  y (null: zeros), routed and h share a type; routed null: no experts.
// pass_through: a choice whose slot is negative stands for x itself, otherwise it adds nothing.  sel as in fi_stream_add.
extern "C" int fi_stream_post(const void* y, long ldy, int y_type, const float* x, const void* routed, long ldr,
                              const int* slot_of, const float* route_w, int top, int pass_through, const float* w_post,
                              const float* w_pre, float* x_out, void* h, long ldh, int h_type, const long long* sel, int rows,
                              int W, int groups, float eps, void* stream) {
  if (rows <= 0) return 0;
  if (W <= 0 || groups <= 0 || W % groups != 0 || h_type < 0 || h_type > 2 || y_type != h_type || top < 0) return -10;
  if ((sel != nullptr && x_out != nullptr) || (routed != nullptr && (route_w == nullptr || top <= 0))) return -10;
  if (w_post == nullptr || (y == nullptr && routed == nullptr) || (w_pre != nullptr && h == nullptr)) return -10;
  StreamParams p = {};
  p.y = y; p.ldy = ldy; p.y_type = y_type; p.x = x; p.routed = routed; p.ldr = ldr; p.slot_of = slot_of; p.route_w = route_w;
  p.top = top; p.pass_through = pass_through; p.w_post = w_post; p.w_pre = w_pre; p.x_out = x_out; p.h = h; p.ldh = ldh;
  p.h_type = h_type; p.sel = sel; p.rows = rows; p.W = W; p.group = W / groups; p.groups = groups; p.eps = eps;
  const bool vec4 = p.group % 4 == 0 && ldh % 4 == 0 && ldy % 4 == 0 && ldr % 4 == 0 && aligned(y, 16) && aligned(x, 16) &&
                    aligned(x_out, 16) && aligned(h, 16) && aligned(routed, 16) && aligned(w_post, 16) && aligned(w_pre, 16);
  return dispatch<kPost>(p, vec4, reinterpret_cast<cudaStream_t>(stream));
}
