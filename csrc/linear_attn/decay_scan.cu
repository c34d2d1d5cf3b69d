// Linear attention with decays, in two forms.  Per head, with state S [d, dv] (32-bit, one slot per sequence):
//
//   channel decays, bonus    y = q S + (sum_i q_i u_i k_i) v,  then  S[i, :] <- w_i S[i, :] + k_i v      (q: the projection r)
//                            ln w_i = -e^(z_i + w0_i) for every key channel i
//   scalar decays, skip      S <- a S + (h k) v (outer product),  then  y = q S + D v                    (q: C, k: B, v: x)
//                            h = softplus(z + bias), ln a = -rate h for every head; B and C belong to groups of heads, and
//                            x, B and C come out of a short causal convolution with bias and SiLU
//
// All arithmetic is 32-bit.
//
//   decay_scan_kernel   portions of prompts: the columns of S never interact, so a warp owns a few columns and walks its
//                       sequence's tokens with its share of S in registers.  Lanes split the d rows 16 ways, the partial
//                       outputs of four tokens are reduced together.  Operands of the next tokens are fetched as raw values
//                       while the present ones are processed, then turned into what the recurrence reads and staged in
//                       shared memory.  Products run as packed pairs (fma.rn.f32x2).
//                       Few long sequences are cut into segments that run side by side: a first pass leaves every segment's end
//                       state from a zero start and the product of its decays, decay_chain_kernel turns those into start states
//                       (and the sequence's last state), and a second pass computes the outputs.
//   decay_step_kernel   one token per sequence (decode): reads and writes the state once; the first form ends with the
//                       per-head norm, weight and gate, the second starts with its convolution.
//   conv_silu_kernel    the convolution of portions: a thread owns channels and slides along a tile of tokens
//   part_norm_kernel    norm over equal parts of a row with weight and SiLU gate (before or after the norm)
//
// The convolution's last inputs live in a ring of `taps` rows per slot, position p in row p % taps.  A decode step writes
// its own row and reads the others; a portion's ring is read and written by the tile that starts it.
// A sequence whose first position is 0 starts from a zero state and zero inputs whatever its slot holds.
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../common/launch.cuh"
#include "recur.cuh"

namespace {
using namespace fi::recur;

enum Kind : int { kChannel = 0, kScalar = 1 };

struct ScanParams {
  const void* q;          // [T, ldq]: r, or C; head (or group) h at columns h * d
  const void* k;          // [T, ldk]: k, or B
  const void* v;          // [T, ldv]: v, or x; head h at columns h * dv
  const float* z;         // [T, ldz]: kChannel H * d decays, kScalar H step sizes
  const float* zb;        // kChannel: w0 [H * d]; kScalar: bias [H]
  const float* u;         // kChannel: bonus [H * d]; kScalar: skip D [H]
  const float* rate;      // kScalar: [H]
  float* pool;            // [slots, H, d, dv]
  const int* slots;       // [B]
  const int* cu_q;        // [B + 1] (scan)
  const int* seq_lens;    // [B] length after this step
  float* o;               // [T, H, dv] (scan; step of kScalar)
  const int* seg_base;    // [B + 1] segments before each sequence, or null: sequences in one piece
  float* seg_state;       // [segments, H, d, dv] end states from zero, then start states
  float* seg_decay;       // [segments, H, d] products of decays (kScalar: the first of each row)
  int seg_len, B;
  // step
  const void* xbc;        // kScalar: [B, ldq] raw x (H * dv) | B (G * d) | C (G * d)
  const float* conv;      // [taps, C]
  const float* conv_b;    // [C]
  float* ring;            // [slots, taps, C]
  const float* norm_w;    // kChannel: [H * dv]
  const void* gate;       // kChannel: [B, ldg]
  void* out;              // kChannel: [B, H * dv]
  long ldq, ldk, ldv, ldz, ldg;
  int vec4, H, G, d, dv, C, taps, type, out_type, num_slots;
  float eps;
};

constexpr int kWarps = 8;

template <int R, int C, int KIND>
struct ScanShape {
  static constexpr int kTok = R <= 8 ? 16 : (R <= 16 ? 8 : 4);     // tokens staged at a time
  static constexpr int D = 16 * R;                                 // padded rows: q = k = 0 there, the state stays 0
  static constexpr int COLS = kWarps * 2 * C;
  static constexpr int NB = (D + 127) / 128;                       // warps that stage one token
  static constexpr int kRows = KIND == kChannel ? 3 : 2;           // staged rows per token: q, k (, decay)
  static constexpr int kFloats = 2 * kTok * (kRows * D + COLS + 4) + 2 * D;
};

// The sequence (or segment) that index i of a running count belongs to.
__device__ __forceinline__ int find_seq(const int* base, int B, int i) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (base[mid] <= i) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// R rows per lane (16 R >= d), C columns per lane (a warp: 2 C columns, a block: 16 C); T: storage of q, k and v.
// OUT: outputs are computed; otherwise (first pass over segments) only states and products of decays.
template <int R, int C, int KIND, typename T, bool OUT>
__global__ void __launch_bounds__(kWarps * 32) decay_scan_kernel(const ScanParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  using L = ScanShape<R, C, KIND>;
  constexpr int kTok = L::kTok, D = L::D, COLS = L::COLS, NB = L::NB;
  constexpr int NQ = kTok * D / 4 / 256;                     // groups of four values per thread
  constexpr int NVAL = (kTok * COLS / 4 + 255) / 256;
  static_assert(NQ * 256 * 4 == kTok * D, "every thread stages whole groups");
  extern __shared__ __align__(16) float smem[];
  float* sq = smem;                                          // [2][kTok][D]
  float* sk = sq + 2 * kTok * D;
  float* sw = sk + 2 * kTok * D;                             // kChannel
  float* sv = smem + 2 * kTok * D * L::kRows;                // [2][kTok][COLS]
  float* sx = sv + 2 * kTok * COLS;                          // [2][kTok][4]: kChannel bonus shares, kScalar decay
  float* c0 = sx + 2 * kTok * 4;                             // [D] w0
  float* c1 = c0 + D;                                        // [D] u
  const int slices = (p.dv + COLS - 1) / COLS;
  const int head = blockIdx.x / slices, slice = blockIdx.x % slices;
  const bool cut = p.seg_base != nullptr;
  const int b = cut ? find_seq(p.seg_base, p.B, blockIdx.y) : blockIdx.y;
  const int s0 = cut ? (static_cast<int>(blockIdx.y) - p.seg_base[b]) * p.seg_len : 0;
  const int t_begin = p.cu_q[b] + s0, n = cut ? min(p.cu_q[b + 1] - t_begin, p.seg_len) : p.cu_q[b + 1] - t_begin;
  if (n <= 0) return;
  const int slot = p.slots[b];
  if (slot < 0 || slot >= p.num_slots) return;
  const bool fresh = !OUT || (!cut && p.seq_lens[b] == n);      // starts from zero
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rg = lane & 15, cg = lane >> 4;
  const int col0 = slice * COLS + (warp * 2 + cg) * C;     // first of this lane's columns
  const long piece = static_cast<long>(cut ? blockIdx.y : slot) * p.H + head;
  float* S0 = (cut ? p.seg_state : p.pool) + piece * p.d * p.dv;
  const int group = head / (p.H / p.G);

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

  Raw4<T> rq[NQ], rk[NQ], rv[NVAL];         // raw values of the next kTok tokens
  Raw4<float> rz[KIND == kChannel ? NQ : 1];
  float rdt[KIND == kScalar ? NQ : 1];
  const T* gq = reinterpret_cast<const T*>(p.q) + group * p.d;
  const T* gk = reinterpret_cast<const T*>(p.k) + group * p.d;
  const T* gv = reinterpret_cast<const T*>(p.v) + head * p.dv + slice * COLS;
  const float* gz = p.z + (KIND == kChannel ? head * p.d : head);
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int e = (i * 256 + threadIdx.x) * 4, tok = e / D, ch = e % D;
      const int left = t0 + tok < n ? p.d - ch : 0;
      const long t = t_begin + t0 + tok;
      if constexpr (OUT) rq[i] = load4(gq + t * p.ldq + ch, left, p.vec4);
      rk[i] = load4(gk + t * p.ldk + ch, left, p.vec4);
      if constexpr (KIND == kChannel) rz[i] = load4(gz + t * p.ldz + ch, left, p.vec4);
      else rdt[i] = t0 + tok < n ? gz[t * p.ldz] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < NVAL; ++i) {
      const int e = (i * 256 + threadIdx.x) * 4, tok = e / COLS, c = e % COLS;
      const int left = (tok < kTok && t0 + tok < n) ? p.dv - slice * COLS - c : 0;
      rv[i] = load4(gv + static_cast<long>(t_begin + t0 + tok) * p.ldv + c, left, p.vec4);
    }
  };
  const float dt_bias = KIND == kScalar ? p.zb[head] : 0.f, rate = KIND == kScalar ? p.rate[head] : 0.f;
  const float skip = KIND == kScalar ? p.u[head] : 0.f;
  // tokens past the end are staged with q = k = 0 and a decay of one: they leave the state as it is
  auto stage = [&](int buf, int t0) {
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int e = (i * 256 + threadIdx.x) * 4, tok = e / D, ch = e % D;
      const bool live = t0 + tok < n;
      float qa[4], ka[4];
      if constexpr (OUT) expand4(rq[i], p.type, qa);          // zeros beyond the last channel and the last token
      expand4(rk[i], p.type, ka);
      const int at = (buf * kTok + tok) * D + ch;
      if constexpr (KIND == kChannel) {
        float za[4], wa[4], bonus = 0.f;
        expand4(rz[i], kFp32, za);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          wa[j] = live && ch + j < p.d ? decay_exp(-__expf(za[j] + c0[ch + j])) : 1.f;
          if constexpr (OUT) bonus = fmaf(qa[j] * c1[ch + j], ka[j], bonus);
        }
        *reinterpret_cast<float4*>(sw + at) = make_float4(wa[0], wa[1], wa[2], wa[3]);
        if constexpr (OUT) {
          constexpr int kLanes = D / 4 < 32 ? D / 4 : 32;      // neighbouring lanes that hold one token
#pragma unroll
          for (int m = kLanes / 2; m > 0; m >>= 1) bonus += __shfl_xor_sync(0xffffffffu, bonus, m);
          if ((lane & (kLanes - 1)) == 0) sx[(buf * kTok + tok) * 4 + ch / 128] = bonus;
        }
      } else {
        const float dt = softplusf(rdt[i] + dt_bias);
#pragma unroll
        for (int j = 0; j < 4; ++j) ka[j] *= dt;
        if (ch == 0) sx[(buf * kTok + tok) * 4] = live ? decay_exp(-rate * dt) : 1.f;
      }
      if constexpr (OUT) *reinterpret_cast<float4*>(sq + at) = make_float4(qa[0], qa[1], qa[2], qa[3]);
      *reinterpret_cast<float4*>(sk + at) = make_float4(ka[0], ka[1], ka[2], ka[3]);
    }
#pragma unroll
    for (int i = 0; i < NVAL; ++i) {
      const int e = (i * 256 + threadIdx.x) * 4, tok = e / COLS, c = e % COLS;
      if (tok < kTok) {
        float v4[4];
        expand4(rv[i], p.type, v4);
        *reinterpret_cast<float4*>(sv + (buf * kTok + tok) * COLS + c) = make_float4(v4[0], v4[1], v4[2], v4[3]);
      }
    }
  };

  if constexpr (KIND == kChannel)
    for (int c = threadIdx.x; c < D; c += 256) {
      c0[c] = c < p.d ? p.zb[head * p.d + c] : 0.f;
      c1[c] = c < p.d ? p.u[head * p.d + c] : 0.f;
    }
  f2 prod[!OUT && KIND == kChannel ? R / 2 : 1];             // products of decays: rows of this lane, or one number
#pragma unroll
  for (int i = 0; i < (!OUT && KIND == kChannel ? R / 2 : 1); ++i) prod[i] = pack2(1.f, 1.f);
  fetch(0);
  __syncthreads();
  stage(0, 0);
  __syncthreads();
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
        const int tok = buf * kTok + tq + u;
        f2 dec = pack2(0.f, 0.f);
        if constexpr (KIND == kScalar) {
          const float a = sx[tok * 4];
          dec = pack2(a, a);
          if constexpr (!OUT) prod[0] = mul2(prod[0], dec);
        }
#pragma unroll
        for (int c = 0; c < C; ++c) {
          acc[c] = pack2(0.f, 0.f);
          const float x = sv[tok * COLS + (warp * 2 + cg) * C + c];
          vv[c] = pack2(x, x);
        }
#pragma unroll
        for (int i4 = 0; i4 < R / 4; ++i4) {
          const int at = tok * D + i4 * 64 + rg * 4;
          const float4 q4 = OUT ? *reinterpret_cast<const float4*>(sq + at) : make_float4(0.f, 0.f, 0.f, 0.f);
          const float4 k4 = *reinterpret_cast<const float4*>(sk + at);
          const f2 qp[2] = {pack2(q4.x, q4.y), pack2(q4.z, q4.w)};
          const f2 kp[2] = {pack2(k4.x, k4.y), pack2(k4.z, k4.w)};
          f2 wp[2] = {dec, dec};
          if constexpr (KIND == kChannel) {
            const float4 w4 = *reinterpret_cast<const float4*>(sw + at);
            wp[0] = pack2(w4.x, w4.y);
            wp[1] = pack2(w4.z, w4.w);
            if constexpr (!OUT) {
              prod[i4 * 2] = mul2(prod[i4 * 2], wp[0]);
              prod[i4 * 2 + 1] = mul2(prod[i4 * 2 + 1], wp[1]);
            }
          }
#pragma unroll
          for (int j = 0; j < 2; ++j) {
#pragma unroll
            for (int c = 0; c < C; ++c) {
              const f2 old = S[i4 * 2 + j][c];
              const f2 s = fma2(wp[j], old, mul2(kp[j], vv[c]));
              S[i4 * 2 + j][c] = s;
              if constexpr (OUT) acc[c] = fma2(qp[j], KIND == kChannel ? old : s, acc[c]);
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
      if constexpr (!OUT) return;
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
          const int u = (base + i) / C, c = (base + i) % C, tok = buf * kTok + tq + u;
          if (tq + u < here && col0 + c < p.dv) {
            float g = skip;
            if constexpr (KIND == kChannel) {
              g = 0.f;
#pragma unroll
              for (int j = 0; j < NB; ++j) g += sx[tok * 4 + j];
            }
            p.o[(static_cast<long>(t_begin + t0 + tq + u) * p.H + head) * p.dv + col0 + c] =
                fmaf(g, sv[tok * COLS + (warp * 2 + cg) * C + c], part[i]);
          }
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

  if (OUT && cut) return;                   // decay_chain_kernel has stored the sequence's state
  if constexpr (!OUT) {
    if (slice == 0 && warp == 0 && cg == 0) {
      float* dst = p.seg_decay + piece * p.d;
      float a, bb;
      if constexpr (KIND == kScalar) {
        unpack2(prod[0], a, bb);
        if (rg == 0) dst[0] = a;
      } else {
#pragma unroll
        for (int i = 0; i < R / 2; ++i) {
          const int row = (i >> 1) * 64 + rg * 4 + (i & 1) * 2;
          unpack2(prod[i], a, bb);
          if (row < p.d) dst[row] = a;
          if (row + 1 < p.d) dst[row + 1] = bb;
        }
      }
    }
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

// Start states of segments from their end states and decays, and the sequences' last states.  Block: (256 groups of VEC state
// values, head, sequence).
template <int VEC, int KIND>
__global__ void __launch_bounds__(256) decay_chain_kernel(const ScanParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  const int head = blockIdx.y, b = blockIdx.z, slot = p.slots[b];
  const int at = (blockIdx.x * 256 + threadIdx.x) * VEC, size = p.d * p.dv;
  const int n = p.cu_q[b + 1] - p.cu_q[b];
  if (at >= size || n <= 0 || slot < 0 || slot >= p.num_slots) return;
  float* pool = p.pool + (static_cast<long>(slot) * p.H + head) * size + at;
  const int row = KIND == kChannel ? at / p.dv : 0;          // a group lies in one row
  float S[VEC];
  auto load = [](const float* src, float* v) {
    if constexpr (VEC == 4) expand4(load4(src, 4, 1), kFp32, v); else v[0] = src[0];
  };
  auto store = [](float* dst, const float* v) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]); else dst[0] = v[0];
  };
#pragma unroll
  for (int e = 0; e < VEC; ++e) S[e] = 0.f;
  if (p.seq_lens[b] != n) load(pool, S);
  const int end = p.seg_base[b + 1];
  constexpr int U = 4;                      // segments whose values are in flight together
  for (int g0 = p.seg_base[b]; g0 < end; g0 += U) {
    float u[U][VEC], w[U];
#pragma unroll
    for (int i = 0; i < U; ++i) {
      const long piece = static_cast<long>(min(g0 + i, end - 1)) * p.H + head;
      load(p.seg_state + piece * size + at, u[i]);
      w[i] = p.seg_decay[piece * p.d + row];
    }
#pragma unroll
    for (int i = 0; i < U; ++i) {
      if (g0 + i >= end) break;
      store(p.seg_state + (static_cast<long>(g0 + i) * p.H + head) * size + at, S);
#pragma unroll
      for (int e = 0; e < VEC; ++e) S[e] = fmaf(w[i], S[e], u[i][e]);
    }
  }
  store(pool, S);
}

__device__ __forceinline__ float block_sum(float v, float* red) {      // 256 threads; red[8] is free again after the next barrier
  for (int m = 16; m > 0; m >>= 1) v += __shfl_xor_sync(0xffffffffu, v, m);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) s += red[w];
  return s;
}

// One token per sequence.  Block: one (head, sequence); thread: VEC columns of every RY-th row.
template <int VEC, int KIND>
__global__ void __launch_bounds__(256, 3) decay_step_kernel(const ScanParams p) {
  fi::pdl_launch_dependents();
  {                                        // the state comes from memory: ask for it while the predecessor ends
    const int s = p.slots[blockIdx.y];
    if (p.seq_lens[blockIdx.y] > 1 && s >= 0 && s < p.num_slots) {
      const float* S = p.pool + (static_cast<long>(s) * p.H + blockIdx.x) * p.d * p.dv;
      for (int i = threadIdx.x * 32; i < p.d * p.dv; i += 256 * 32) fi::prefetch_l2(S + i);
    }
  }
  fi::pdl_wait();
  extern __shared__ __align__(16) float smem[];
  __shared__ float red[2][8];
  const int head = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int len = p.seq_lens[b], slot = p.slots[b], d = p.d, dv = p.dv;
  const long orow = static_cast<long>(b) * p.H * dv + static_cast<long>(head) * dv;
  if (len <= 0 || slot < 0 || slot >= p.num_slots) {       // padded row of a decode bucket
    for (int j = tid; j < dv; j += 256) {
      if constexpr (KIND == kChannel) st_any(p.out, orow + j, p.out_type, 0.f);
      else p.o[orow + j] = 0.f;
    }
    return;
  }
  float* sq = smem;                 // [d]
  float* sk = sq + d;               // [d]
  float* sw = sk + d;               // [d] (kChannel)
  float* sv = sw + d;               // [dv]
  float* so = sv + dv;              // [ry][dv] partial outputs
  const int nx = (dv + VEC - 1) / VEC;                     // threads across the columns (<= 256)
  const int ry_n = 256 / nx, cx = tid % nx, ry = tid / nx;
  const bool fresh = len == 1;
  float* S = p.pool + (static_cast<long>(slot) * p.H + head) * d * dv;
  const int per = p.H / p.G, group = head / per;
  constexpr int U = 8;                  // rows whose loads are in flight together; the first ones while the operands are prepared
  float s[U][VEC];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int i = 0; i < U; ++i) {
      const int r = r0 + i * ry_n;
#pragma unroll
      for (int e = 0; e < VEC; ++e) s[i][e] = 0.f;
      if (!fresh && r < d) {
        const float* row = S + static_cast<long>(r) * dv + cx * VEC;
        if constexpr (VEC == 4) {
          const float4 x = *reinterpret_cast<const float4*>(row);
          s[i][0] = x.x; s[i][1] = x.y; s[i][2] = x.z; s[i][3] = x.w;
        } else {
          s[i][0] = row[0];
        }
      }
    }
  };
  if (ry < ry_n) fetch(ry);
  float decay = 1.f, g = 0.f;       // kScalar: decay and skip; kChannel: g is the bonus
  if constexpr (KIND == kChannel) {
    for (int c = tid; c < d; c += 256) {
      const long at = static_cast<long>(group) * d + c;
      const float r = ld_any(p.q, b * p.ldq + at, p.type), k = ld_any(p.k, b * p.ldk + at, p.type);
      const int hc = head * d + c;
      sq[c] = r;
      sk[c] = k;
      sw[c] = decay_exp(-__expf(p.z[b * p.ldz + hc] + p.zb[hc]));
      g = fmaf(r * p.u[hc], k, g);
    }
    for (int c = tid; c < dv; c += 256) sv[c] = ld_any(p.v, b * p.ldv + static_cast<long>(head) * dv + c, p.type);
    g = block_sum(g, red[0]);       // its barrier also publishes the operands
  } else {
    const float dt = softplusf(p.z[b * p.ldz + head] + p.zb[head]);
    decay = decay_exp(-p.rate[head] * dt);
    g = p.u[head];
    const int pos = len - 1, taps = p.taps;
    float* ring = p.ring + static_cast<long>(slot) * taps * p.C;
    const int inner = p.H * dv, at = pos % taps;
#pragma unroll 2
    for (int c = tid; c < 2 * d + dv; c += 256) {
      const int ch = c < d ? inner + (p.G + group) * d + c : (c < 2 * d ? inner + group * d + c - d : head * dv + c - 2 * d);
      const float now = ld_any(p.xbc, b * p.ldq + ch, p.type);
      float y = fmaf(p.conv[static_cast<long>(taps - 1) * p.C + ch], now, p.conv_b[ch]);
      auto back = [&](int j) {             // j tokens back
        if (j >= taps || pos - j < 0) return;
        const int row = at >= j ? at - j : at - j + taps;
        y = fmaf(p.conv[static_cast<long>(taps - 1 - j) * p.C + ch], ring[static_cast<long>(row) * p.C + ch], y);
      };
#pragma unroll
      for (int j = 1; j < 4; ++j) back(j);
      for (int j = 4; j < taps; ++j) back(j);
      if (c >= 2 * d || head % per == 0) ring[static_cast<long>(at) * p.C + ch] = now;
      y *= sigmoidf(y);
      if (c < d) sq[c] = y;
      else if (c < 2 * d) sk[c - d] = dt * y;
      else sv[c - 2 * d] = y;
    }
    __syncthreads();
  }
  if (ry < ry_n) {
    float v[VEC], o[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      v[e] = sv[cx * VEC + e];
      o[e] = 0.f;
    }
    for (int r0 = ry; r0 < d; r0 += U * ry_n) {
      if (r0 != ry) fetch(r0);
#pragma unroll
      for (int i = 0; i < U; ++i) {
        const int r = r0 + i * ry_n;
        if (r < d) {
          float* row = S + static_cast<long>(r) * dv + cx * VEC;
          const float k = sk[r], q = sq[r], w = KIND == kChannel ? sw[r] : decay;
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            const float old = s[i][e];
            s[i][e] = fmaf(w, old, k * v[e]);
            o[e] = fmaf(q, KIND == kChannel ? old : s[i][e], o[e]);
          }
          if constexpr (VEC == 4) *reinterpret_cast<float4*>(row) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
          else row[0] = s[i][0];
        }
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) so[ry * dv + cx * VEC + e] = o[e];
  }
  __syncthreads();
  float ss = 0.f;
  for (int j = tid; j < dv; j += 256) {
    float o = 0.f;
    for (int r = 0; r < ry_n; ++r) o += so[r * dv + j];
    o = fmaf(g, sv[j], o);
    if constexpr (KIND == kScalar) {
      p.o[orow + j] = o;
    } else {
      so[j] = o;                          // row 0 of its own column: nobody else reads it any more
      ss = fmaf(o, o, ss);
    }
  }
  if constexpr (KIND == kChannel) {
    const float inv = 1.f / sqrtf(block_sum(ss, red[1]) / static_cast<float>(dv) + p.eps);
    for (int j = tid; j < dv; j += 256) {
      const long at = static_cast<long>(head) * dv + j;
      float y = so[j] * inv * p.norm_w[at];
      if (p.gate != nullptr) {
        const float z = ld_any(p.gate, b * p.ldg + at, p.type);
        y *= z * sigmoidf(z);
      }
      st_any(p.out, orow + j, p.out_type, y);
    }
  }
}

struct ConvParams {
  const void* x;           // [T, ld]
  const float* w;          // [taps, C]
  const float* bias;       // [C]
  float* ring;             // [slots, taps, C]
  void* out;               // [T, C]
  const int* slots;
  const int* cu_q;
  const int* seq_lens;
  const int* tile_base;    // [B + 1] tiles before each sequence
  long ld;
  int B, C, taps, tile, num_slots, type, out_type;
};

// VEC values of type TYPE (known at compile time: the convolution is bound by its instructions).
template <int VEC, int TYPE>
__device__ __forceinline__ void load_as(const void* p, long i, float* v) {
  if constexpr (TYPE == kFp32) {
    const float* f = reinterpret_cast<const float*>(p) + i;
    if constexpr (VEC == 4) expand4(load4(f, 4, 1), kFp32, v); else v[0] = f[0];
  } else if constexpr (VEC == 4) {
    expand4(load4(reinterpret_cast<const uint16_t*>(p) + i, 4, 1), TYPE, v);
  } else {
    v[0] = ld_any(p, i, TYPE);
  }
}
template <int VEC, int TYPE>
__device__ __forceinline__ void store_as(void* p, long i, const float* v) {
  if constexpr (VEC == 1) {
    st_any(p, i, TYPE, v[0]);
  } else if constexpr (TYPE == kFp32) {
    *reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + i) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    uint32_t w[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      if constexpr (TYPE == kBf16) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
        w[e] = *reinterpret_cast<const uint32_t*>(&h);
      } else {
        const __half2 h = __floats2half2_rn(v[2 * e], v[2 * e + 1]);
        w[e] = *reinterpret_cast<const uint32_t*>(&h);
      }
    }
    *reinterpret_cast<uint2*>(reinterpret_cast<uint16_t*>(p) + i) = make_uint2(w[0], w[1]);
  }
}

// KT >= taps: registers of the sliding window (leading taps of weight zero).  IN, OUT: types of x and out.
template <int KT, int VEC, int IN, int OUT>
__global__ void __launch_bounds__(128, KT > 4 ? 1 : 8) conv_silu_kernel(const ConvParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  int lo = 0, hi = p.B - 1;
  while (lo < hi) {                        // the sequence this tile belongs to
    const int mid = (lo + hi + 1) >> 1;
    if (p.tile_base[mid] <= static_cast<int>(blockIdx.x)) lo = mid; else hi = mid - 1;
  }
  const int b = lo, i0 = (static_cast<int>(blockIdx.x) - p.tile_base[b]) * p.tile;
  const int t_begin = p.cu_q[b], n = p.cu_q[b + 1] - t_begin;
  const int pos0 = p.seq_lens[b] - n, slot = p.slots[b];
  const int c = (blockIdx.y * 128 + threadIdx.x) * VEC;
  if (i0 < 0 || i0 >= n || slot < 0 || slot >= p.num_slots || c >= p.C) return;
  const int taps = p.taps;
  float* ring = p.ring + static_cast<long>(slot) * taps * p.C + c;
  const long x0 = t_begin * p.ld + c;
  float a[KT][VEC], seq[KT + 3][VEC], bias[VEC];             // seq: the KT - 1 inputs before the present four, then those
#pragma unroll
  for (int j = 0; j < KT; ++j) {
    const int tap = j - (KT - taps);
    load_as<VEC, kFp32>(p.w, static_cast<long>(max(tap, 0)) * p.C + c, a[j]);
    if (tap < 0)
#pragma unroll
      for (int e = 0; e < VEC; ++e) a[j][e] = 0.f;
  }
  // loads take no branches, so that they are in flight together
  if (i0 > 0) {                            // a tile holds at least taps tokens
#pragma unroll
    for (int j = 0; j + 1 < KT; ++j) load_as<VEC, IN>(p.x, x0 + max(i0 - KT + 1 + j, 0) * p.ld, seq[j]);
  } else {
#pragma unroll
    for (int j = 0; j + 1 < KT; ++j) {
      const int i = j - KT + 1;
#pragma unroll
      for (int e = 0; e < VEC; ++e) seq[j][e] = 0.f;
      if (-i < taps && pos0 + i >= 0) load_as<VEC, kFp32>(ring, static_cast<long>((pos0 + i) % taps) * p.C, seq[j]);
    }
  }
  load_as<VEC, kFp32>(p.bias, c, bias);
  const int i_end = min(n, i0 + p.tile);
  for (int i = i0; i < i_end; i += 4) {
#pragma unroll
    for (int u = 0; u < 4; ++u) load_as<VEC, IN>(p.x, x0 + min(i + u, i_end - 1) * p.ld, seq[KT - 1 + u]);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (i + u >= i_end) break;
      float y[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = bias[e];
#pragma unroll
      for (int j = 0; j < KT; ++j)
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = fmaf(a[j][e], seq[j + u][e], y[e]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] *= sigmoidf(y[e]);
      store_as<VEC, OUT>(p.out, static_cast<long>(t_begin + i + u) * p.C + c, y);
    }
#pragma unroll
    for (int j = 0; j + 1 < KT; ++j)
#pragma unroll
      for (int e = 0; e < VEC; ++e) seq[j][e] = seq[j + 4][e];
  }
  if (i0 == 0)
    for (int i = max(0, n - taps); i < n; ++i) {
      float v[VEC];
      load_as<VEC, IN>(p.x, x0 + i * p.ld, v);
      store_as<VEC, kFp32>(ring, static_cast<long>((pos0 + i) % taps) * p.C, v);
    }
}

template <int KT, int VEC>
int launch_conv(const ConvParams& p, int tiles, cudaStream_t s) {
  const dim3 g(tiles, (p.C + 128 * VEC - 1) / (128 * VEC));
  auto kern = p.type == kFp32 ? (p.out_type == kFp32   ? conv_silu_kernel<KT, VEC, kFp32, kFp32>
                                 : p.out_type == kBf16 ? conv_silu_kernel<KT, VEC, kFp32, kBf16>
                                                       : conv_silu_kernel<KT, VEC, kFp32, kFp16>)
              : p.type == kBf16 ? conv_silu_kernel<KT, VEC, kBf16, kBf16>
                                : conv_silu_kernel<KT, VEC, kFp16, kFp16>;
  return static_cast<int>(fi::launch_kernel(kern, g, dim3(128), 0, s, 0, p));
}

struct NormParams {
  const float* x;      // [T, parts * n]
  const void* gate;    // [T, ldg] or null
  const float* w;      // [parts * n]
  void* out;           // [T, parts * n]
  long rows, ldg;      // rows: T * parts
  int parts, n, gate_type, gate_first, out_type;
  float eps;
};

// A row of n values per TPR threads (16, 32 or 256), NV groups of four each (NV = 0: any n, one value at a time, read twice).
template <int TPR, int NV>
__global__ void __launch_bounds__(256) part_norm_kernel(const NormParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  __shared__ float red[8];
  constexpr int per = 256 / TPR;
  long row = static_cast<long>(blockIdx.x) * per + (per == 1 ? 0 : static_cast<int>(threadIdx.x) / TPR);
  if (TPR >= 32 && row >= p.rows) return;
  const bool live = row < p.rows;          // half warps leave together
  if (!live) row = p.rows - 1;
  const int tid = per == 1 ? threadIdx.x : threadIdx.x % TPR;
  const long t = row / p.parts;
  const int part = static_cast<int>(row % p.parts), n = p.n;
  const float* x = p.x + row * n;
  const float* w = p.w + static_cast<long>(part) * n;
  const long grow = t * p.ldg + static_cast<long>(part) * n;
  float ss = 0.f;
  auto total = [&]() {
#pragma unroll
    for (int m = TPR < 32 ? TPR / 2 : 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    if constexpr (TPR > 32) {
      if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
      __syncthreads();
      ss = 0.f;
#pragma unroll
      for (int i = 0; i < TPR / 32; ++i) ss += red[i];
    }
  };
  if constexpr (NV > 0) {
    float v[NV][4], g[NV][4];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * 4;
#pragma unroll
      for (int e = 0; e < 4; ++e) { v[i][e] = 0.f; g[i][e] = 0.f; }
      if (c < n) {
        const float4 f = *reinterpret_cast<const float4*>(x + c);
        v[i][0] = f.x; v[i][1] = f.y; v[i][2] = f.z; v[i][3] = f.w;
        if (p.gate != nullptr) {
          if (p.gate_type == kFp32) expand4(load4(reinterpret_cast<const float*>(p.gate) + grow + c, 4, 1), kFp32, g[i]);
          else expand4(load4(reinterpret_cast<const uint16_t*>(p.gate) + grow + c, 4, 1), p.gate_type, g[i]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        g[i][e] = p.gate != nullptr ? g[i][e] * sigmoidf(g[i][e]) : 1.f;
        if (p.gate_first) v[i][e] *= g[i][e];
        ss = fmaf(v[i][e], v[i][e], ss);
      }
    total();
    const float inv = 1.f / sqrtf(ss / static_cast<float>(n) + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * TPR + tid) * 4;
      if (c >= n || !live) continue;
      const float4 f = *reinterpret_cast<const float4*>(w + c);
      float y[4] = {v[i][0] * inv * f.x, v[i][1] * inv * f.y, v[i][2] * inv * f.z, v[i][3] * inv * f.w};
      if (!p.gate_first)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] *= g[i][e];
      if (p.out_type == kFp32) {
        *reinterpret_cast<float4*>(reinterpret_cast<float*>(p.out) + row * n + c) = make_float4(y[0], y[1], y[2], y[3]);
      } else {
        alignas(8) uint16_t h[4];
#pragma unroll
        for (int e = 0; e < 4; ++e)
          h[e] = p.out_type == kBf16 ? __bfloat16_as_ushort(__float2bfloat16_rn(y[e])) : __half_as_ushort(__float2half_rn(y[e]));
        *reinterpret_cast<uint2*>(reinterpret_cast<uint16_t*>(p.out) + row * n + c) = *reinterpret_cast<const uint2*>(h);
      }
    }
  } else {
    auto gate = [&](int c) {
      if (p.gate == nullptr) return 1.f;
      const float z = ld_any(p.gate, grow + c, p.gate_type);
      return z * sigmoidf(z);
    };
    for (int c = tid; c < n; c += TPR) {
      const float v = x[c] * (p.gate_first ? gate(c) : 1.f);
      ss = fmaf(v, v, ss);
    }
    total();
    const float inv = 1.f / sqrtf(ss / static_cast<float>(n) + p.eps);
    for (int c = tid; c < n; c += TPR) st_any(p.out, row * n + c, p.out_type, x[c] * gate(c) * inv * w[c]);
  }
}

template <int R, int C, int KIND, bool OUT>
int launch_scan(const ScanParams& p, int pieces, cudaStream_t s) {
  using L = ScanShape<R, C, KIND>;
  const dim3 grid(p.H * ((p.dv + L::COLS - 1) / L::COLS), pieces), block(kWarps * 32);
  constexpr int smem = L::kFloats * 4;
  auto kern = p.type == kFp32 ? decay_scan_kernel<R, C, KIND, float, OUT> : decay_scan_kernel<R, C, KIND, uint16_t, OUT>;
  const cudaError_t e = fi::ensure_dynamic_smem(kern, smem);
  if (e != cudaSuccess) return static_cast<int>(e);
  return static_cast<int>(fi::launch_kernel(kern, grid, block, smem, s, 0, p));
}

template <int R, int KIND, bool OUT>
int pick_cols(const ScanParams& p, int B, cudaStream_t s) {
  // wide tiles spend the fewest instructions per element, narrow ones fill the device when there are few sequences
  const long ctas4 = static_cast<long>(B) * p.H * ((p.dv + 63) / 64);
  if constexpr (R <= 8) {
    if (ctas4 >= 192) return launch_scan<R, 4, KIND, OUT>(p, B, s);
  }
  if (ctas4 >= 120) return launch_scan<R, 2, KIND, OUT>(p, B, s);
  return launch_scan<R, 1, KIND, OUT>(p, B, s);
}

template <int KIND, bool OUT>
int dispatch_pass(const ScanParams& p, int pieces, cudaStream_t s) {
  if (p.d <= 64) return pick_cols<4, KIND, OUT>(p, pieces, s);
  if (p.d <= 128) return pick_cols<8, KIND, OUT>(p, pieces, s);
  if (p.d <= 256) return pick_cols<16, KIND, OUT>(p, pieces, s);
  if (p.d <= 512) return launch_scan<32, 1, KIND, OUT>(p, pieces, s);
  return -11;
}

template <int KIND>
int dispatch_scan(const ScanParams& p, int segments, cudaStream_t s) {
  if (p.seg_base == nullptr) return dispatch_pass<KIND, true>(p, p.B, s);
  int rc = dispatch_pass<KIND, false>(p, segments, s);
  if (rc != 0) return rc;
  const bool vec4 = p.dv % 4 == 0 && ((reinterpret_cast<uintptr_t>(p.pool) | reinterpret_cast<uintptr_t>(p.seg_state)) & 15) == 0;
  const int per = 256 * (vec4 ? 4 : 1);
  auto kern = vec4 ? decay_chain_kernel<4, KIND> : decay_chain_kernel<1, KIND>;
  rc = static_cast<int>(fi::launch_kernel(kern, dim3((p.d * p.dv + per - 1) / per, p.H, p.B), dim3(256), 0, s, 0, p));
  return rc != 0 ? rc : dispatch_pass<KIND, true>(p, segments, s);
}

template <int KIND>
int dispatch_step(const ScanParams& p, int B, cudaStream_t s) {
  const bool vec4 = p.dv % 4 == 0 && (reinterpret_cast<uintptr_t>(p.pool) & 15) == 0;
  const int nx = vec4 ? p.dv / 4 : p.dv;
  if (nx > 256) return -11;
  const int smem = (3 * p.d + p.dv + (256 / nx) * p.dv) * 4;
  if (smem > 48 * 1024) return -11;
  auto kern = vec4 ? decay_step_kernel<4, KIND> : decay_step_kernel<1, KIND>;
  return static_cast<int>(fi::launch_kernel(kern, dim3(p.H, B), dim3(256), smem, s, 0, p));
}

bool vec_rows(const ScanParams& p, bool z_rows) {
  const uintptr_t mask = p.type == kFp32 ? 15 : 7;
  return p.d % 4 == 0 && p.dv % 4 == 0 && (p.ldq | p.ldk | p.ldv) % 4 == 0 &&
         ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.k) | reinterpret_cast<uintptr_t>(p.v)) & mask) == 0 &&
         (!z_rows || (p.ldz % 4 == 0 && (reinterpret_cast<uintptr_t>(p.z) & 15) == 0));
}

}  // namespace

// Portions.  kind 0 (channel decays, bonus): q = r, k, v rows of H heads (G = H), z fp32 [T, ldz] (H * d), zb = w0 [H * d],
// u = bonus [H * d], rate unused.  kind 1 (scalar decays, skip): q = C and k = B rows of G groups, v = x of H heads, z fp32
// [T, ldz] (H step sizes), zb = their bias [H], u = D [H], rate [H].  type (0 bf16, 1 fp16, 2 fp32): q, k and v.  pool fp32
// [num_slots, H, d, dv]; o fp32 [T, H, dv].  d <= 512.  seg_base (or null) int32 [B + 1] counts segments of seg_len tokens,
// `segments` its last entry; seg_state fp32 [segments, H, d, dv] and seg_decay fp32 [segments, H, d] are scratch.
extern "C" int fi_decay_scan(int kind, const void* q, long ldq, const void* k, long ldk, const void* v, long ldv, const float* z,
                             long ldz, const float* zb, const float* u, const float* rate, float* pool, const int* slots,
                             const int* cu_q, const int* seq_lens, float* o, const int* seg_base, int seg_len, int segments,
                             float* seg_state, float* seg_decay, int B, int H, int G, int d, int dv, int num_slots, int type,
                             void* stream) {
  if (B <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G != 0 || d <= 0 || dv <= 0 || B > 65535 || type < 0 || type > 2 || (kind != 0 && kind != 1)) return -10;
  if (seg_base != nullptr && (seg_len <= 0 || segments <= 0 || segments > 65535 || seg_state == nullptr || seg_decay == nullptr)) return -10;
  ScanParams p = {};
  p.q = q; p.k = k; p.v = v; p.ldq = ldq; p.ldk = ldk; p.ldv = ldv; p.z = z; p.ldz = ldz; p.zb = zb; p.u = u; p.rate = rate;
  p.pool = pool; p.slots = slots; p.cu_q = cu_q; p.seq_lens = seq_lens; p.o = o; p.H = H; p.G = G; p.d = d; p.dv = dv;
  p.num_slots = num_slots; p.type = type; p.B = B; p.seg_base = seg_base; p.seg_len = seg_len; p.seg_state = seg_state;
  p.seg_decay = seg_decay;
  p.vec4 = vec_rows(p, kind == 0);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return kind == 0 ? dispatch_scan<kChannel>(p, segments, s) : dispatch_scan<kScalar>(p, segments, s);
}

// One token per sequence, channel decays: operands of fi_decay_scan with B rows, then per head norm(o) * norm_w [H * dv] *
// silu(gate) (gate [B, ldg] of `type`, or null) into out [B, H * dv] of out_type.  Rows with seq_lens <= 0 are padding.
extern "C" int fi_decay_step(const void* q, long ldq, const void* k, long ldk, const void* v, long ldv, const float* z, long ldz,
                             const float* w0, const float* u, const void* gate, long ldg, const float* norm_w, float eps, float* pool,
                             const int* slots, const int* seq_lens, void* out, int B, int H, int d, int dv, int num_slots, int type,
                             int out_type, void* stream) {
  if (B <= 0) return 0;
  if (H <= 0 || d <= 0 || dv <= 0 || B > 65535 || type < 0 || type > 2 || out_type < 0 || out_type > 2) return -10;
  ScanParams p = {};
  p.q = q; p.k = k; p.v = v; p.ldq = ldq; p.ldk = ldk; p.ldv = ldv; p.z = z; p.ldz = ldz; p.zb = w0; p.u = u; p.gate = gate;
  p.ldg = ldg; p.norm_w = norm_w; p.eps = eps; p.pool = pool; p.slots = slots; p.seq_lens = seq_lens; p.out = out; p.H = H;
  p.G = H; p.d = d; p.dv = dv; p.num_slots = num_slots; p.type = type; p.out_type = out_type;
  return dispatch_step<kChannel>(p, B, reinterpret_cast<cudaStream_t>(stream));
}

// One token per sequence, scalar decays, convolution included: xbc [B, ld] of `type` = x (H * dv) | B (G * d) | C (G * d) before
// the convolution conv fp32 [taps, channels] with bias; ring fp32 [num_slots, taps, channels]; z fp32 [B, ldz] (H step sizes).
// o fp32 [B, H, dv].
extern "C" int fi_decay_step_conv(const void* xbc, long ld, const float* z, long ldz, const float* bias, const float* rate,
                                  const float* skip, const float* conv, const float* conv_b, int taps, float* ring, float* pool,
                                  const int* slots, const int* seq_lens, float* o, int B, int H, int G, int d, int dv,
                                  int num_slots, int type, void* stream) {
  if (B <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G != 0 || d <= 0 || dv <= 0 || B > 65535 || taps <= 0 || type < 0 || type > 2) return -10;
  ScanParams p = {};
  p.xbc = xbc; p.ldq = ld; p.z = z; p.ldz = ldz; p.zb = bias; p.rate = rate; p.u = skip; p.conv = conv; p.conv_b = conv_b;
  p.taps = taps; p.ring = ring; p.pool = pool; p.slots = slots; p.seq_lens = seq_lens; p.o = o; p.H = H; p.G = G; p.d = d;
  p.dv = dv; p.C = H * dv + 2 * G * d; p.num_slots = num_slots; p.type = type;
  return dispatch_step<kScalar>(p, B, reinterpret_cast<cudaStream_t>(stream));
}

// Convolution with bias and SiLU over portions: x [T, ld] (type) -> out [T, C] (out_type; the same or, from 32-bit, any); w fp32 [taps, C]; ring as above;
// tile_base int32 [B + 1] counts tiles of `tile` tokens (at least taps), n_tiles its last entry.
extern "C" int fi_conv_silu(const void* x, long ld, const float* w, const float* bias, int taps, float* ring, void* out,
                            const int* slots, const int* cu_q, const int* seq_lens, const int* tile_base, int n_tiles, int tile,
                            int B, int C, int num_slots, int type, int out_type, void* stream) {
  if (n_tiles <= 0 || B <= 0) return 0;
  if (C <= 0 || taps <= 0 || taps > 16 || tile < taps || type < 0 || type > 2 || out_type < 0 || out_type > 2 ||
      (type != kFp32 && out_type != type))
    return -10;
  ConvParams p = {};
  p.x = x; p.ld = ld; p.w = w; p.bias = bias; p.taps = taps; p.ring = ring; p.out = out; p.slots = slots; p.cu_q = cu_q;
  p.seq_lens = seq_lens; p.tile_base = tile_base; p.tile = tile; p.B = B; p.C = C; p.num_slots = num_slots; p.type = type;
  p.out_type = out_type;
  const bool vec4 = C % 4 == 0 && ld % 4 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(w) |
                                                   reinterpret_cast<uintptr_t>(bias) | reinterpret_cast<uintptr_t>(ring)) & 15) == 0;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (taps <= 4) return vec4 ? launch_conv<4, 4>(p, n_tiles, s) : launch_conv<4, 1>(p, n_tiles, s);
  if (taps <= 8) return vec4 ? launch_conv<8, 4>(p, n_tiles, s) : launch_conv<8, 1>(p, n_tiles, s);
  return launch_conv<16, 1>(p, n_tiles, s);
}

// out [T, parts * n] = norm over each part of n values of x fp32 [T, parts * n], times w, with a SiLU gate [T, ldg] (or null)
// applied before (gate_first) or after the norm.
extern "C" int fi_part_norm(const float* x, const void* gate, long ldg, int gate_type, int gate_first, const float* w, int parts,
                            void* out, long T, int n, float eps, int out_type, void* stream) {
  if (T <= 0) return 0;
  if (n <= 0 || parts <= 0 || gate_type < 0 || gate_type > 2 || out_type < 0 || out_type > 2) return -10;
  NormParams p = {};
  p.x = x; p.gate = gate; p.ldg = ldg; p.gate_type = gate_type; p.gate_first = gate_first; p.w = w; p.parts = parts; p.out = out;
  p.rows = T * parts; p.n = n; p.eps = eps; p.out_type = out_type;
  const bool vec = n % 4 == 0 && ldg % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(gate) |
                     reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define FI_NORM(TPR, NV)                                                                                               \
  return static_cast<int>(fi::launch_kernel(part_norm_kernel<TPR, NV>, dim3(static_cast<unsigned>((p.rows + 256 / TPR - 1) / (256 / TPR))), \
                                            dim3(256), 0, s, 0, p))
  if (!vec || n > 8192) {
    if (n <= 256) FI_NORM(32, 0);
    FI_NORM(256, 0);
  }
  if (n <= 64) FI_NORM(16, 1);
  if (n <= 128) FI_NORM(32, 1);
  if (n <= 256) FI_NORM(32, 2);
  if (n <= 512) FI_NORM(32, 4);
  if (n <= 1024) FI_NORM(256, 1);
  if (n <= 2048) FI_NORM(256, 2);
  if (n <= 4096) FI_NORM(256, 4);
  FI_NORM(256, 8);
#undef FI_NORM
}
