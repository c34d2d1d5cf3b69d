// HGRN2 linear attention: per head, with state S [d, dv] (32-bit, one slot per sequence),
//
//   f_t = l + (1 - l) sigmoid(z_t + b)       S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T       o_t = S_t^T silu(q_t)
//
// All arithmetic is 32-bit.  The write strength is evaluated directly as (1 - l) sigmoid(-(z + b)) and the forget
// gate as one minus it, so that a gate close to one keeps the full precision of what is written.
//
//   hgrn2_scan_kernel   portions of prompts (also single tokens beside them): the columns of S never interact, so a
//                       warp owns a few columns and walks its sequence's tokens with its share of S in registers.
//                       Lanes split the d rows 16 ways (each lane 4, 8, ... rows), the partial outputs of four
//                       tokens are reduced together.  Gate values of the next 16 tokens (fewer for wide heads) are
//                       fetched while the present ones are processed, then activated and staged in shared memory.  Products run as packed pairs
//                       (fma.rn.f32x2).
//   hgrn2_step_kernel   one token per sequence (decode): reads and writes the state once, 16 bytes per thread and
//                       access, and finishes with the per-head RMS norm.
//   head_norm_kernel    RMS norm of each head's output row (after the scan), optionally times sigmoid of a gate.
// A sequence whose first position is 0 starts from a zero state whatever its slot holds.
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../common/launch.cuh"
#include "recur.cuh"

namespace {

using namespace fi::recur;
__device__ __forceinline__ float ld(const void* p, long i, int type) { return ld_any(p, i, type); }
__device__ __forceinline__ void st(void* p, long i, int type, float v) { st_any(p, i, type, v); }

struct Hgrn2Params {
  const void* q;          // [T, ldq] projection outputs: head h at columns h * d
  const void* f;          // [T, ldf]
  const void* v;          // [T, ldv]: head h at columns h * dv
  const float* f_bias;    // [H * d]
  const float* lower;     // [H * d]
  float* pool;            // [slots, H, d, dv]
  const int* slots;       // [B]
  const int* cu_q;        // [B + 1] (scan)
  const int* seq_lens;    // [B] length after this step
  float* o;               // scan: [T, H, dv]
  const float* norm_w;    // step: [dv]
  void* out;              // step: [B, H * dv]
  long ldq, ldf, ldv;
  int vec4;               // rows of q, f and v start on whole groups of four values
  int H, d, dv, qv_type, f_type, out_type, num_slots;
  float eps;
};

constexpr int kWarps = 8;

// R rows per lane (16 R >= d), C columns per lane (a warp: 2 C columns, a block: 16 C); T: storage of q and v.
template <int R, int C, typename T>
__global__ void __launch_bounds__(kWarps * 32) hgrn2_scan_kernel(const Hgrn2Params p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  constexpr int kTok = R <= 8 ? 16 : (R <= 16 ? 8 : 4);     // tokens staged at a time
  constexpr int D = 16 * R;                 // padded rows: q = k = 0 there, the state stays 0
  constexpr int COLS = kWarps * 2 * C;
  constexpr int NQ = (kTok * D / 4 + 255) / 256;             // groups of four values per thread
  constexpr int NVAL = (kTok * COLS / 4 + 255) / 256;
  __shared__ __align__(16) float sq[2][kTok][D];
  __shared__ __align__(16) float sk[2][kTok][D];
  __shared__ __align__(16) float sv[2][kTok][COLS];
  __shared__ float open_gate[D], gate_bias[D];
  const int slices = (p.dv + COLS - 1) / COLS;
  const int head = blockIdx.x / slices, slice = blockIdx.x % slices;
  const int b = blockIdx.y;
  const int t_begin = p.cu_q[b], n = p.cu_q[b + 1] - t_begin;
  if (n <= 0) return;
  const int slot = p.slots[b];
  if (slot < 0 || slot >= p.num_slots) return;
  const bool fresh = p.seq_lens[b] == n;    // the portion starts at position 0
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rg = lane & 15, cg = lane >> 4;
  const int col0 = slice * COLS + (warp * 2 + cg) * C;     // first of this lane's columns
  float* S0 = p.pool + (static_cast<long>(slot) * p.H + head) * p.d * p.dv;

  // rows of this lane: 64 i4 + 4 rg + e, pairs (e = 0, 1) and (2, 3)
  f2 S[R / 2][C];
#pragma unroll
  for (int i = 0; i < R / 2; ++i) {
    const int row = (i >> 1) * 64 + rg * 4 + (i & 1) * 2;
#pragma unroll
    for (int c = 0; c < C; ++c) {
      float a = 0.f, bb = 0.f;
      if (!fresh && col0 + c < p.dv) {
        if (row < p.d) a = S0[static_cast<long>(row) * p.dv + col0 + c];
        if (row + 1 < p.d) bb = S0[static_cast<long>(row + 1) * p.dv + col0 + c];
      }
      S[i][c] = pack2(a, bb);
    }
  }

  Raw4<T> rq[NQ], rv[NVAL];                 // raw values of the next kTok tokens
  Raw4<float> rf[NQ];
  const T* gq = reinterpret_cast<const T*>(p.q) + head * p.d;
  const T* gv = reinterpret_cast<const T*>(p.v) + head * p.dv + slice * COLS;
  const float* gf = reinterpret_cast<const float*>(p.f) + head * p.d;
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int e = (i * 256 + threadIdx.x) * 4, tok = e / D, ch = e % D;
      const int left = (tok < kTok && t0 + tok < n) ? p.d - ch : 0;
      const long t = t_begin + t0 + tok;
      rq[i] = load4(gq + t * p.ldq + ch, left, p.vec4);
      rf[i] = load4(gf + t * p.ldf + ch, left, p.vec4);
    }
#pragma unroll
    for (int i = 0; i < NVAL; ++i) {
      const int e = (i * 256 + threadIdx.x) * 4, tok = e / COLS, c = e % COLS;
      const int left = (tok < kTok && t0 + tok < n) ? p.dv - slice * COLS - c : 0;
      rv[i] = load4(gv + static_cast<long>(t_begin + t0 + tok) * p.ldv + c, left, p.vec4);
    }
  };
  // tokens past the end are staged with q = k = 0: they leave the state as it is
  auto stage = [&](int buf, int t0) {
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int e = (i * 256 + threadIdx.x) * 4, tok = e / D, ch = e % D;
      if (tok < kTok) {
        float zq[4], zf[4], qa[4], ka[4];
        expand4(rq[i], p.qv_type, zq);
        expand4(rf[i], kFp32, zf);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          qa[j] = 0.f; ka[j] = 0.f;
          if (ch + j < p.d && t0 + tok < n) {
            qa[j] = zq[j] * sigmoidf(zq[j]);
            ka[j] = open_gate[ch + j] * sigmoidf(-(zf[j] + gate_bias[ch + j]));
          }
        }
        *reinterpret_cast<float4*>(&sq[buf][tok][ch]) = make_float4(qa[0], qa[1], qa[2], qa[3]);
        *reinterpret_cast<float4*>(&sk[buf][tok][ch]) = make_float4(ka[0], ka[1], ka[2], ka[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < NVAL; ++i) {
      const int e = (i * 256 + threadIdx.x) * 4, tok = e / COLS, c = e % COLS;
      if (tok < kTok) {
        float v4[4];
        expand4(rv[i], p.qv_type, v4);
        *reinterpret_cast<float4*>(&sv[buf][tok][c]) = make_float4(v4[0], v4[1], v4[2], v4[3]);
      }
    }
  };

  for (int c = threadIdx.x; c < D; c += 256) {
    open_gate[c] = c < p.d ? 1.f - p.lower[head * p.d + c] : 0.f;
    gate_bias[c] = c < p.d ? p.f_bias[head * p.d + c] : 0.f;
  }
  fetch(0);
  __syncthreads();
  stage(0, 0);
  __syncthreads();
  const f2 one2 = pack2(1.f, 1.f), neg2 = pack2(-1.f, -1.f);
  for (int t0 = 0, it = 0; t0 < n; t0 += kTok, ++it) {
    const int buf = it & 1;
    const bool more = t0 + kTok < n;
    if (more) fetch(t0 + kTok);
    const int here = min(kTok, n - t0);
    auto four_tokens = [&](int tq) {
      float part[4 * C];                    // partial outputs [token][column] of this lane's rows
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        f2 acc[C], vv[C];
        const int tok = tq + u;
#pragma unroll
        for (int c = 0; c < C; ++c) {
          acc[c] = pack2(0.f, 0.f);
          const float x = sv[buf][tok][(warp * 2 + cg) * C + c];
          vv[c] = pack2(x, x);
        }
#pragma unroll
        for (int i4 = 0; i4 < R / 4; ++i4) {
          const float4 q4 = *reinterpret_cast<const float4*>(&sq[buf][tok][i4 * 64 + rg * 4]);
          const float4 k4 = *reinterpret_cast<const float4*>(&sk[buf][tok][i4 * 64 + rg * 4]);
          const f2 qp[2] = {pack2(q4.x, q4.y), pack2(q4.z, q4.w)};
          const f2 kp[2] = {pack2(k4.x, k4.y), pack2(k4.z, k4.w)};
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const f2 fp = fma2(kp[j], neg2, one2);
#pragma unroll
            for (int c = 0; c < C; ++c) {
              const f2 s = fma2(fp, S[i4 * 2 + j][c], mul2(kp[j], vv[c]));
              S[i4 * 2 + j][c] = s;
              acc[c] = fma2(qp[j], s, acc[c]);
            }
          }
        }
#pragma unroll
        for (int c = 0; c < C; ++c) {
          float lo, hi;
          unpack2(acc[c], lo, hi);
          part[u * C + c] = lo + hi;
        }
      }
      // sum over the 16 row lanes; each halving step keeps half of the values on either side
      int base = 0, width = 4 * C;
#pragma unroll
      for (int m = 8; m > 0; m >>= 1) {
        if (width > 1) {
          const int half = width / 2;
          const bool up = (rg & m) != 0;
#pragma unroll
          for (int i = 0; i < 2 * C; ++i) {
            if (i < half) {
              const float send = up ? part[i] : part[i + half];
              const float keep = up ? part[i + half] : part[i];
              part[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
            }
          }
          if (up) base += half;
          width = half;
        } else {
          part[0] += __shfl_xor_sync(0xffffffffu, part[0], m);
        }
      }
      // after the halving steps a lane holds `width` values starting at index `base` of [4][C]; when there are
      // fewer values than row lanes the last steps were plain sums and one lane of each set stores
      constexpr int kSteps = 4 * C >= 16 ? 4 : (4 * C == 8 ? 3 : 2);
      constexpr int kLeft = (4 * C) >> kSteps;
      const bool writer = (rg & ((1 << (4 - kSteps)) - 1)) == 0;
      if (writer) {
#pragma unroll
        for (int i = 0; i < kLeft; ++i) {
          const int u = (base + i) / C, c = (base + i) % C;
          if (tq + u < here && col0 + c < p.dv)
            p.o[(static_cast<long>(t_begin + t0 + tq + u) * p.H + head) * p.dv + col0 + c] = part[i];
        }
      }
    };
    if (here == kTok) {                     // full stage: straight-line code, the sums of one group of four tokens
#pragma unroll                              // overlap the products of the next
      for (int tq = 0; tq < kTok; tq += 4) four_tokens(tq);
    } else {
      for (int tq = 0; tq < here; tq += 4) four_tokens(tq);
    }
    if (more) stage(buf ^ 1, t0 + kTok);
    __syncthreads();
  }

#pragma unroll
  for (int i = 0; i < R / 2; ++i) {
    const int row = (i >> 1) * 64 + rg * 4 + (i & 1) * 2;
#pragma unroll
    for (int c = 0; c < C; ++c) {
      float a, bb;
      unpack2(S[i][c], a, bb);
      if (col0 + c < p.dv) {
        if (row < p.d) S0[static_cast<long>(row) * p.dv + col0 + c] = a;
        if (row + 1 < p.d) S0[static_cast<long>(row + 1) * p.dv + col0 + c] = bb;
      }
    }
  }
}

// One token per sequence.  Block: one (head, sequence); thread: VEC columns of every RY-th row.
template <int VEC>
__global__ void __launch_bounds__(256, 3) hgrn2_step_kernel(const Hgrn2Params p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  extern __shared__ float smem[];
  const int head = blockIdx.x, b = blockIdx.y;
  const int len = p.seq_lens[b], slot = p.slots[b];
  const long orow = static_cast<long>(b) * p.H * p.dv + static_cast<long>(head) * p.dv;
  if (len <= 0 || slot < 0 || slot >= p.num_slots) {      // padded row of a decode bucket
    for (int j = threadIdx.x; j < p.dv; j += blockDim.x) st(p.out, orow + j, p.out_type, 0.f);
    return;
  }
  float* sq = smem;                 // [d]
  float* sk = sq + p.d;             // [d]
  float* so = sk + p.d;             // [ry][dv] partial outputs
  const int nx = (p.dv + VEC - 1) / VEC;                  // threads across the columns (<= 256)
  const int ry_n = 256 / nx;
  for (int c = threadIdx.x; c < p.d; c += blockDim.x) {
    const float zq = ld(p.q, b * p.ldq + head * p.d + c, p.qv_type);
    const float zf = ld(p.f, b * p.ldf + head * p.d + c, p.f_type) + p.f_bias[head * p.d + c];
    sq[c] = zq * sigmoidf(zq);
    sk[c] = (1.f - p.lower[head * p.d + c]) * sigmoidf(-zf);
  }
  __syncthreads();
  const bool fresh = len == 1;
  const int cx = threadIdx.x % nx, ry = threadIdx.x / nx;
  float* S = p.pool + (static_cast<long>(slot) * p.H + head) * p.d * p.dv;
  if (ry < ry_n) {
    float v[VEC], o[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      v[e] = ld(p.v, b * p.ldv + head * p.dv + cx * VEC + e, p.qv_type);
      o[e] = 0.f;
    }
    constexpr int U = 8;                  // rows whose loads are in flight together
    for (int r0 = ry; r0 < p.d; r0 += U * ry_n) {
      float s[U][VEC];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = r0 + u * ry_n;
#pragma unroll
        for (int e = 0; e < VEC; ++e) s[u][e] = 0.f;
        if (!fresh && r < p.d) {
          const float* row = S + static_cast<long>(r) * p.dv + cx * VEC;
          if constexpr (VEC == 4) {
            const float4 x = *reinterpret_cast<const float4*>(row);
            s[u][0] = x.x; s[u][1] = x.y; s[u][2] = x.z; s[u][3] = x.w;
          } else {
            s[u][0] = row[0];
          }
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = r0 + u * ry_n;
        if (r < p.d) {
          float* row = S + static_cast<long>(r) * p.dv + cx * VEC;
          const float k = sk[r], q = sq[r], f = 1.f - k;
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            s[u][e] = fmaf(f, s[u][e], k * v[e]);
            o[e] = fmaf(q, s[u][e], o[e]);
          }
          if constexpr (VEC == 4) *reinterpret_cast<float4*>(row) = make_float4(s[u][0], s[u][1], s[u][2], s[u][3]);
          else row[0] = s[u][0];
        }
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) so[ry * p.dv + cx * VEC + e] = o[e];
  }
  __syncthreads();
  __shared__ float red[8];
  float ss = 0.f;
  for (int j = threadIdx.x; j < p.dv; j += blockDim.x) {
    float o = 0.f;
    for (int r = 0; r < ry_n; ++r) o += so[r * p.dv + j];
    so[j] = o;                      // row 0 of its own column: nobody else reads it any more
    ss += o * o;
  }
  for (int m = 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int w = 0; w < 8; ++w) tot += red[w];
  const float inv = 1.f / sqrtf(tot / static_cast<float>(p.dv) + p.eps);
  for (int j = threadIdx.x; j < p.dv; j += blockDim.x) st(p.out, orow + j, p.out_type, so[j] * inv * p.norm_w[j]);
}

// RMS norm of rows of length dv (fp32 in), one warp per row; with `gate` (row of token t at t * ldg, H heads of dv) the
// result is multiplied by sigmoid(gate).
__global__ void __launch_bounds__(256) head_norm_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                        const void* __restrict__ gate, long ldg, int gate_type, int H,
                                                        void* __restrict__ out, long rows, int dv, float eps, int type) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  const long row = static_cast<long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (row >= rows) return;
  const int lane = threadIdx.x & 31;
  const float* src = x + row * dv;
  const long grow = gate != nullptr ? (row / H) * ldg + (row % H) * dv : 0;
  float ss = 0.f;
  if ((dv & 3) == 0 && dv <= 512 && ((grow | ldg) & 3) == 0 && (reinterpret_cast<uintptr_t>(gate) & 15) == 0) {
    float4 v[4];
    float gt[4][4];                         // raw gates, in flight together with the row
    if (gate != nullptr) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int c = (i * 32 + lane) * 4;
        if (c < dv) {
          if (gate_type == kFp32) expand4(load4(reinterpret_cast<const float*>(gate) + grow + c, 4, 1), kFp32, gt[i]);
          else expand4(load4(reinterpret_cast<const uint16_t*>(gate) + grow + c, 4, 1), gate_type, gt[i]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = (i * 32 + lane) * 4;
      v[i] = c < dv ? *reinterpret_cast<const float4*>(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    for (int m = 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    const float inv = 1.f / sqrtf(ss / static_cast<float>(dv) + eps);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = (i * 32 + lane) * 4;
      if (c < dv) {
        const float4 g = *reinterpret_cast<const float4*>(w + c);
        float y[4] = {v[i].x * inv * g.x, v[i].y * inv * g.y, v[i].z * inv * g.z, v[i].w * inv * g.w};
        if (gate != nullptr)
#pragma unroll
          for (int e = 0; e < 4; ++e) y[e] *= sigmoidf(gt[i][e]);
        if (type == kFp32) {
          *reinterpret_cast<float4*>(reinterpret_cast<float*>(out) + row * dv + c) = make_float4(y[0], y[1], y[2], y[3]);
        } else {
          alignas(8) uint16_t h[4];
          for (int e = 0; e < 4; ++e)
            h[e] = type == kBf16 ? __bfloat16_as_ushort(__float2bfloat16_rn(y[e])) : __half_as_ushort(__float2half_rn(y[e]));
          *reinterpret_cast<uint2*>(reinterpret_cast<uint16_t*>(out) + row * dv + c) = *reinterpret_cast<uint2*>(h);
        }
      }
    }
    return;
  }
  for (int c = lane; c < dv; c += 32) ss += src[c] * src[c];
  for (int m = 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(dv) + eps);
  for (int c = lane; c < dv; c += 32) {
    float y = src[c] * inv * w[c];
    if (gate != nullptr) y *= sigmoidf(ld(gate, grow + c, gate_type));
    st(out, row * dv + c, type, y);
  }
}

template <int R, int C>
int launch_scan(const Hgrn2Params& p, int B, cudaStream_t s) {
  constexpr int COLS = kWarps * 2 * C;
  const dim3 grid(p.H * ((p.dv + COLS - 1) / COLS), B), block(kWarps * 32);
  if (p.qv_type == kFp32) return static_cast<int>(fi::launch_kernel(hgrn2_scan_kernel<R, C, float>, grid, block, 0, s, 0, p));
  return static_cast<int>(fi::launch_kernel(hgrn2_scan_kernel<R, C, uint16_t>, grid, block, 0, s, 0, p));
}

template <int R>
int pick_cols(const Hgrn2Params& p, int B, cudaStream_t s) {
  // wide tiles spend the fewest instructions per element, narrow ones fill the device when there are few sequences
  const long ctas4 = static_cast<long>(B) * p.H * ((p.dv + 63) / 64);
  if constexpr (R <= 8) {
    if (ctas4 >= 192) return launch_scan<R, 4>(p, B, s);
  }
  if (ctas4 >= 120) return launch_scan<R, 2>(p, B, s);
  return launch_scan<R, 1>(p, B, s);
}

}  // namespace

// Portions of sequences.  q, v: type qv_type (0 bf16, 1 fp16, 2 fp32), f: fp32 (f_type 2), rows of pitch ldq / ldf / ldv;
// f_bias, lower: fp32 [H * d]; pool: fp32 [num_slots, H, d, dv]; slots, seq_lens: int32 [B]; cu_q: int32 [B + 1];
// o: fp32 [T, H, dv].
extern "C" int fi_hgrn2_scan(const void* q, long ldq, const void* f, long ldf, const void* v, long ldv,
                             const float* f_bias, const float* lower, float* pool, const int* slots, const int* cu_q,
                             const int* seq_lens, float* o, int B, int H, int d, int dv, int num_slots, int qv_type,
                             int f_type, void* stream) {
  if (B <= 0) return 0;
  if (H <= 0 || d <= 0 || dv <= 0 || B > 65535 || qv_type < 0 || qv_type > 2 || f_type != kFp32) return -10;
  Hgrn2Params p = {};
  p.q = q; p.f = f; p.v = v; p.ldq = ldq; p.ldf = ldf; p.ldv = ldv; p.f_bias = f_bias; p.lower = lower; p.pool = pool;
  p.slots = slots; p.cu_q = cu_q; p.seq_lens = seq_lens; p.o = o; p.H = H; p.d = d; p.dv = dv; p.num_slots = num_slots;
  p.qv_type = qv_type;
  const uintptr_t mask = qv_type == kFp32 ? 15 : 7;
  p.vec4 = d % 4 == 0 && dv % 4 == 0 && ldq % 4 == 0 && ldf % 4 == 0 && ldv % 4 == 0 &&
           ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(v)) & mask) == 0 && (reinterpret_cast<uintptr_t>(f) & 15) == 0;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (d <= 64) return pick_cols<4>(p, B, s);
  if (d <= 128) return pick_cols<8>(p, B, s);
  if (d <= 256) return pick_cols<16>(p, B, s);
  if (d <= 512) return launch_scan<32, 1>(p, B, s);
  return -11;
}

// RMS norm of every head's row: x fp32 [rows, dv] -> out [rows, dv] (type 0 bf16, 1 fp16, 2 fp32), w fp32 [dv].  gate
// (or null): rows [rows / H, >= H * dv] of pitch ldg and gate_type; out is multiplied by sigmoid(gate).
extern "C" int fi_head_norm(const float* x, const float* w, const void* gate, long ldg, int gate_type, int H, void* out,
                            long rows, int dv, float eps, int type, void* stream) {
  if (rows <= 0) return 0;
  if (dv <= 0 || H <= 0 || type < 0 || type > 2 || gate_type < 0 || gate_type > 2 || (reinterpret_cast<uintptr_t>(x) & 15) != 0 ||
      (reinterpret_cast<uintptr_t>(w) & 15) != 0 || (reinterpret_cast<uintptr_t>(out) & 7) != 0)
    return -10;
  return static_cast<int>(fi::launch_kernel(head_norm_kernel, dim3(static_cast<unsigned>((rows + 7) / 8)), dim3(256), 0,
                                            reinterpret_cast<cudaStream_t>(stream), 0, x, w, gate, ldg, gate_type, H, out, rows, dv, eps,
                                            type));
}

// One token per sequence, norm included.  Same operands as fi_hgrn2_scan; norm_w: fp32 [dv]; out: [B, H * dv] of type
// out_type.  Rows with seq_lens <= 0 are padding: their output is zero and no state is touched.
extern "C" int fi_hgrn2_step(const void* q, long ldq, const void* f, long ldf, const void* v, long ldv,
                             const float* f_bias, const float* lower, float* pool, const int* slots, const int* seq_lens,
                             const float* norm_w, float eps, void* out, int B, int H, int d, int dv, int num_slots,
                             int qv_type, int f_type, int out_type, void* stream) {
  if (B <= 0) return 0;
  if (H <= 0 || d <= 0 || dv <= 0 || B > 65535 || qv_type < 0 || qv_type > 2 || f_type < 0 || f_type > 2 ||
      out_type < 0 || out_type > 2)
    return -10;
  Hgrn2Params p = {};
  p.q = q; p.f = f; p.v = v; p.ldq = ldq; p.ldf = ldf; p.ldv = ldv; p.f_bias = f_bias; p.lower = lower; p.pool = pool;
  p.slots = slots; p.seq_lens = seq_lens; p.norm_w = norm_w; p.eps = eps; p.out = out; p.H = H; p.d = d; p.dv = dv;
  p.num_slots = num_slots; p.qv_type = qv_type; p.f_type = f_type; p.out_type = out_type;
  const bool vec4 = dv % 4 == 0 && (reinterpret_cast<uintptr_t>(pool) & 15) == 0;
  const int nx = vec4 ? dv / 4 : dv;
  if (nx > 256) return -11;
  const int smem = (2 * d + (256 / nx) * dv) * 4;
  if (smem > 48 * 1024) return -11;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (vec4) return static_cast<int>(fi::launch_kernel(hgrn2_step_kernel<4>, dim3(H, B), dim3(256), smem, s, 0, p));
  return static_cast<int>(fi::launch_kernel(hgrn2_step_kernel<1>, dim3(H, B), dim3(256), smem, s, 0, p));
}
