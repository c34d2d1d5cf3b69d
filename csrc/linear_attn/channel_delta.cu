// Gated delta rule with one decay per head and key channel.  Per head, with state S [d, dv] (32-bit, one slot per
// sequence), after a short causal convolution and SiLU on q, k and v:
//
//   q^ = q / |q| * d^-1/2,   k^ = k / |k|,   g = exp(-exp(A) softplus(z + bias)),   beta = sigmoid(b)
//   S <- diag(g) S;   u = beta (v - S^T k^);   S <- S + k^ u^T;   o = S^T q^
//
// q and k may have fewer heads than v (head h reads q / k head h / (H / G)).  All arithmetic is 32-bit.
//
// Portions of prompts run in chunks of 16 tokens.  With E_i the product of the decays from the chunk's start through
// token i (per channel), a chunk's writes are u_i = beta_i (v_i - S_0^T (E_i k_i) - sum_{j<i} a_ij u_j) with
// a_ij = sum_c k_i k_j E_i / E_j, so they solve a unit lower-triangular system, U = U0 - W S_0, and its outputs are
// o = (E q) S_0 + P U = (E q - P W) S_0 + P U0 with p_ij = sum_c q_i k_j E_i / E_j (j <= i).
//
//   delta_chunk_kernel   everything that does not depend on the state, for all chunks in parallel: convolutions, unit
//                        vectors, decays, a_ij and p_ij, the solved W and U0, Q = E q - P W and P U0.  Ratios E_i / E_j
//                        are running products of decays from j to i: at most one, and nothing is divided.
//   delta_scan_kernel    chunk after chunk: [U; o] = [U0; P U0] + [-W; Q] S, S <- E_16 S + sum_j (E_16 / E_j) k_j u_j^T.
//                        A block owns some columns of S, each warp (or half of one) a range of its rows, and each lane
//                        one or two columns of those in registers, so the operand rows are read as broadcasts and a
//                        product needs no exchange between lanes; the row ranges' partial sums meet in shared memory,
//                        first those of U, then those of o.  Operands arrive by bulk copies.
//   delta_step_kernel    one token per sequence (decode): convolution, unit vectors, decays, state, per-head norm and
//                        output gate in one pass that reads and writes the state once.
//
// The last taps - 1 convolution inputs of a sequence live in a ring of `taps` rows per slot: position p in row p % taps.
// A step writes its own row and reads the others, so blocks that share q / k channels never race.
// A sequence whose first position is 0 starts from a zero state and zero inputs whatever its slot holds.
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../common/launch.cuh"
#include "../common/ptx.cuh"
#include "recur.cuh"

namespace {
using namespace fi::recur;

constexpr int kTok = 16;              // tokens per chunk
constexpr float kUnitEps = 1e-6f;

struct DeltaParams {
  const void* qkv;        // [T, ld]: q (G * d) | k (G * d) | v (H * dv)
  const float* z;         // [T, ldz]: decay projection (H * d)
  const float* b;         // [T, ldb]: write strength projection (H)
  const float* conv;      // [C, taps], last column = current token
  const float* rate;      // [H]: exp(A)
  const float* bias;      // [H * d]
  float* pool;            // [slots, H, d, dv]
  float* ring;            // [slots, taps, C]
  const int* slots;       // [B]
  const int* cu_q;        // [B + 1] (portions)
  const int* seq_lens;    // [B] length after this step
  const int* chunk_base;  // [B + 1] chunks before each sequence (portions)
  float* work;            // [chunks, H, work_stride]
  float* o;               // portions: [T, H, dv]
  const float* norm_w;    // step: [dv]
  const void* gate;       // step: [B, ldg] (H * dv) or null
  void* out;              // step: [B, H * dv]
  long ld, ldz, ldb, ldg, work_stride;
  int B, H, G, d, dv, dp, dvp, C, taps, num_slots, n_chunks, gate_type, out_type, vec_o;
  float eps, q_scale;
};

// work block of a (chunk, head), in floats: -W [16][dp] | Q [16][dp] | (E_16 / E) k [16][dp] | E_16 [dp] |
// groups of 16 columns [dvp / 16] of U0 [16 tokens][16] | P U0 [16 tokens][16]
__host__ __device__ inline long work_floats(int dp, int dvp) { return 49l * dp + 32l * dvp; }

// TAPS: convolution length known at compile time (0: any).
template <typename T, int TAPS>
__global__ void __launch_bounds__(256, 3) delta_chunk_kernel(const DeltaParams p) {
  // no early launch of the scan: its few long-lived blocks would pile up on the multiprocessors that drain first
  fi::pdl_wait();
  extern __shared__ __align__(128) float smem[];
  const int chunk = blockIdx.x, head = blockIdx.y, tid = threadIdx.x;
  int lo = 0, hi = p.B - 1;            // the sequence this chunk belongs to
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.chunk_base[mid] <= chunk) lo = mid; else hi = mid - 1;
  }
  const int b = lo;
  const int t0 = (chunk - p.chunk_base[b]) * kTok;
  const int t_begin = p.cu_q[b], n = p.cu_q[b + 1] - t_begin;
  const int valid = min(kTok, n - t0);
  const int slot = p.slots[b];
  if (valid <= 0 || slot < 0 || slot >= p.num_slots) return;
  const int pos0 = p.seq_lens[b] - n;  // position of the portion's first token
  const int d = p.d, dv = p.dv, dp = p.dp, taps = TAPS > 0 ? TAPS : p.taps, hist = taps - 1;
  const int sp = (d + 3) & ~3;         // pitch of the key-channel rows
  const int width = 2 * d + dv;
  const int kvh = head / (p.H / p.G);
  float* sq = smem;                    // [16][sp] activated q (not yet unit vectors)
  float* sk = sq + kTok * sp;          // [16][sp]
  float* sg = sk + kTok * sp;          // [16][sp] decays
  float* skd = sg + kTok * sp;         // [16][sp] E k
  float* sqd = skd + kTok * sp;        // [16][sp] E q
  float* sA = sqd + kTok * sp;         // [16][16]
  float* sP = sA + 256;                // [16][16]
  float* sb = sP + 256;                // [16]
  float* sf = sb + 16;                 // [32] factors that make q (and its scale) and k unit vectors
  float* sv = sf + 32;                 // [16][dv]
  float* work = p.work + (static_cast<long>(chunk) * p.H + head) * p.work_stride;

  // ---- convolutions, activations and decays: an item is one channel over the chunk's tokens
  const T* qkv = reinterpret_cast<const T*>(p.qkv) + (t_begin + t0) * p.ld;
  const float* ring = p.ring + static_cast<long>(slot) * taps * p.C;
  const float rate = p.rate[head];
  for (int c = tid; c < width + d; c += 256) {
    if (c < width) {
      const int ch = c < d ? kvh * d + c : (c < 2 * d ? p.G * d + kvh * d + c - d : 2 * p.G * d + head * dv + c - 2 * d);
      auto input = [&](int r) -> float {         // token t0 + r of the portion (r may be negative)
        if (r >= 0) {
          const float x = to_f(qkv[min(r, valid - 1) * p.ld + ch]);
          return r < valid ? x : 0.f;
        }
        if (t0 > 0) return to_f(qkv[r * p.ld + ch]);      // (chunks are longer than the convolution)
        const int pos = pos0 + r;
        return pos >= 0 ? ring[(pos % taps) * p.C + ch] : 0.f;
      };
      float y[kTok];
      if constexpr (TAPS > 0) {
        float x[kTok + TAPS - 1], w[TAPS];
#pragma unroll
        for (int r = 0; r < kTok + TAPS - 1; ++r) x[r] = input(r - (TAPS - 1));
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = p.conv[static_cast<long>(ch) * TAPS + j];
#pragma unroll
        for (int t = 0; t < kTok; ++t) {
          y[t] = w[0] * x[t];
#pragma unroll
          for (int j = 1; j < TAPS; ++j) y[t] = fmaf(w[j], x[t + j], y[t]);
        }
      } else {
#pragma unroll
        for (int t = 0; t < kTok; ++t) y[t] = 0.f;
        for (int j = 0; j < taps; ++j) {
          const float w = p.conv[static_cast<long>(ch) * taps + j];
#pragma unroll
          for (int t = 0; t < kTok; ++t) y[t] = fmaf(w, input(t + j - hist), y[t]);
        }
      }
      float* dst = c < d ? sq + c : (c < 2 * d ? sk + c - d : sv + c - 2 * d);
      const int pitch = c < 2 * d ? sp : dv;
#pragma unroll
      for (int t = 0; t < kTok; ++t) dst[t * pitch] = t < valid ? y[t] * sigmoidf(y[t]) : 0.f;
    } else {
      const int cg = c - width;
      const float bias = p.bias[head * d + cg];
      const float* z = p.z + (t_begin + t0) * p.ldz + head * d + cg;
      float zz[kTok];
#pragma unroll
      for (int t = 0; t < kTok; ++t) zz[t] = z[min(t, valid - 1) * p.ldz];
#pragma unroll
      for (int t = 0; t < kTok; ++t) sg[t * sp + cg] = t < valid ? decay_exp(-rate * softplusf(zz[t] + bias)) : 1.f;
    }
  }
  for (int i = tid; i < kTok * (sp - d); i += 256) {       // channels that only fill up the last group of four
    const int at = (i / (sp - d)) * sp + d + i % (sp - d);
    sq[at] = 0.f; sk[at] = 0.f; sg[at] = 0.f;
  }
  if (tid < kTok) sb[tid] = tid < valid ? sigmoidf(p.b[(t_begin + t0 + tid) * p.ldb + head]) : 0.f;
  __syncthreads();
  const int warp = tid >> 5, lane = tid & 31;
  {
    float ss[4];                                           // rows warp, warp + 8 of q, then of k
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float* row = (i < 2 ? sq : sk) + (warp + 8 * (i & 1)) * sp;
      ss[i] = 0.f;
      for (int c = lane * 4; c < sp; c += 128) {
        const float4 v = *reinterpret_cast<const float4*>(row + c);
        ss[i] += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      }
    }
#pragma unroll
    for (int m = 16; m > 0; m >>= 1)
#pragma unroll
      for (int i = 0; i < 4; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], m);
    if (lane < 4) {
      const float t = lane == 0 ? ss[0] : lane == 1 ? ss[1] : lane == 2 ? ss[2] : ss[3];
      sf[(lane >> 1) * 16 + warp + 8 * (lane & 1)] = (lane < 2 ? p.q_scale : 1.f) / sqrtf(t + kUnitEps);
    }
  }
  __syncthreads();
  // ---- running products of decays, forward (E q, E k, E_16) and backward (E_16 / E k)
  for (int it = tid; it < 2 * dp; it += 256) {
    const bool back = it >= dp;
    const int c = back ? it - dp : it;
    if (c >= d) {                                          // rows of S that only fill up the lanes' groups
      float* out = work + (back ? 32l : 0l) * dp + c;
#pragma unroll
      for (int t = 0; t < kTok; ++t) {
        out[t * dp] = 0.f;
        if (!back) out[(16 + t) * dp] = 0.f;
      }
      if (!back) work[48l * dp + c] = 0.f;
    } else if (!back) {
      float e = 1.f;
#pragma unroll
      for (int t = 0; t < kTok; ++t) {
        e *= sg[t * sp + c];
        sqd[t * sp + c] = sq[t * sp + c] * e * sf[t];
        skd[t * sp + c] = sk[t * sp + c] * e * sf[16 + t];
      }
      work[48l * dp + c] = e;
    } else {
      float r = 1.f;
      float* out = work + 32l * dp + c;
#pragma unroll
      for (int t = kTok - 1; t >= 0; --t) {
        out[t * dp] = sk[t * sp + c] * r * sf[16 + t];
        r *= sg[t * sp + c];
      }
    }
  }
  // ---- a_ij (lanes 0-15 end with rows i) and p_ij (lanes 16-31) of two columns j per warp
#pragma unroll 1
  for (int side = 0; side < 2; ++side) {
    const int j = side == 0 ? warp : kTok - 1 - warp;
    float v[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) v[i] = 0.f;
    for (int c = lane * 4; c < sp; c += 128) {
      const float4 k4 = *reinterpret_cast<const float4*>(sk + j * sp + c);
      f2 w0 = pack2(k4.x, k4.y), w1 = pack2(k4.z, k4.w);
#pragma unroll
      for (int i = 0; i < kTok; ++i) {
        if (i < j) continue;
        float x, y;
        if (i > j) {
          const float4 g4 = *reinterpret_cast<const float4*>(sg + i * sp + c);
          const float4 a4 = *reinterpret_cast<const float4*>(sk + i * sp + c);
          w0 = mul2(w0, pack2(g4.x, g4.y));
          w1 = mul2(w1, pack2(g4.z, g4.w));
          unpack2(fma2(pack2(a4.x, a4.y), w0, mul2(pack2(a4.z, a4.w), w1)), x, y);
          v[i] += x + y;
        }
        const float4 q4 = *reinterpret_cast<const float4*>(sq + i * sp + c);
        unpack2(fma2(pack2(q4.x, q4.y), w0, mul2(pack2(q4.z, q4.w), w1)), x, y);
        v[16 + i] += x + y;
      }
    }
#pragma unroll
    for (int m = 16; m > 0; m >>= 1) {
      const bool up = (lane & m) != 0;
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        if (i < m) {
          const float send = up ? v[i] : v[i + m];
          const float keep = up ? v[i + m] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
        }
      }
    }
    const int i = lane & 15;
    const float scaled = v[0] * sf[16 + j] * sf[(lane < 16 ? 16 : 0) + i];
    if (lane < 16) sA[i * 16 + j] = scaled;
    else sP[i * 16 + j] = scaled;
  }
  __syncthreads();
  // ---- solve for one column of W or U0 per thread
  for (int c = tid; c < d + dv; c += 256) {
    const float* src = c < d ? skd + c : sv + c - d;
    const int pitch = c < d ? sp : dv;
    float x[kTok];
#pragma unroll
    for (int i = 0; i < kTok; ++i) {
      asm volatile("" ::: "memory");                       // keeps the coefficients from being loaded all at once
      float r = src[i * pitch];
#pragma unroll
      for (int j4 = 0; j4 < (i + 3) / 4; ++j4) {           // coefficients from i on are zero
        const float4 a4 = *reinterpret_cast<const float4*>(sA + i * 16 + j4 * 4);
        r = fmaf(-a4.x, x[j4 * 4], r);
        if (j4 * 4 + 1 < i) r = fmaf(-a4.y, x[j4 * 4 + 1], r);
        if (j4 * 4 + 2 < i) r = fmaf(-a4.z, x[j4 * 4 + 2], r);
        if (j4 * 4 + 3 < i) r = fmaf(-a4.w, x[j4 * 4 + 3], r);
      }
      x[i] = sb[i] * r;
    }
    float* out = c < d ? work + c : work + 49l * dp + ((c - d) >> 4) * 512 + ((c - d) & 15);
    const int step = c < d ? dp : 16;
#pragma unroll
    for (int i = 0; i < kTok; ++i) {                       // P W or P U0
      asm volatile("" ::: "memory");
      float r = 0.f;
#pragma unroll
      for (int j4 = 0; j4 <= i / 4; ++j4) {
        const float4 p4 = *reinterpret_cast<const float4*>(sP + i * 16 + j4 * 4);
        r = fmaf(p4.x, x[j4 * 4], r);
        if (j4 * 4 + 1 <= i) r = fmaf(p4.y, x[j4 * 4 + 1], r);
        if (j4 * 4 + 2 <= i) r = fmaf(p4.z, x[j4 * 4 + 2], r);
        if (j4 * 4 + 3 <= i) r = fmaf(p4.w, x[j4 * 4 + 3], r);
      }
      out[i * step] = c < d ? -x[i] : x[i];
      out[(16 + i) * step] = c < d ? sqd[i * sp + c] - r : r;
    }
  }
  for (int i = tid; i < (p.dvp - dv) * 32; i += 256) {
    const int cc = dv + i / 32;
    work[49l * dp + (cc >> 4) * 512 + (i & 31) * 16 + (cc & 15)] = 0.f;
  }
}

__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(fi::smem_u32(dst)),
               "l"(src), "r"(bytes), "r"(fi::smem_u32(bar))
               : "memory");
}

// WARPS x LR row ranges of RPL rows (dp == WARPS LR RPL); a lane owns CPL columns of its range, a block 32 / LR * CPL.
template <int RPL, int LR, int CPL, int WARPS, int STAGES>
__global__ void __launch_bounds__(WARPS * 32) delta_scan_kernel(const DeltaParams p, int* status) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  constexpr int THREADS = WARPS * 32;
  constexpr int PARTS = WARPS * LR, DP = PARTS * RPL;
  constexpr int COLS = 32 / LR * CPL;
  constexpr int kBase = 49 * DP;                           // stage offset of U0 | P U0
  constexpr int kStage = kBase + 32 * COLS;
  constexpr int NP = RPL / 2;                              // pairs of rows per lane
  extern __shared__ __align__(128) float smem[];
  float* part = smem + STAGES * kStage;                    // [PARTS][16][COLS] partial products of U, then of o
  float* su = part + PARTS * 16 * COLS;                    // [16][COLS] U
  __shared__ uint64_t full[STAGES];
  const int slices = p.dvp / COLS;
  const int head = blockIdx.x / slices, slice = blockIdx.x % slices, b = blockIdx.y;
  const int t_begin = p.cu_q[b], n = p.cu_q[b + 1] - t_begin;
  const int slot = p.slots[b];
  if (n <= 0 || slot < 0 || slot >= p.num_slots) return;
  const int first = p.chunk_base[b], chunks = (n + kTok - 1) / kTok;
  const int seq_len = p.seq_lens[b];
  const bool fresh = seq_len == n;                         // the portion starts at position 0
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int range = warp * LR + lane / (32 / LR);          // this lane's rows: [range * RPL, ..)
  const int lcol = lane % (32 / LR) * CPL;                 // first of this lane's columns inside the block
  const int col0 = slice * COLS + lcol;
  float* S0 = p.pool + (static_cast<long>(slot) * p.H + head) * p.d * p.dv;

  if (tid == 0) {
    for (int s = 0; s < STAGES; ++s) fi::mbar_init(&full[s], 1);
    fi::mbar_fence_init();
  }
  __syncthreads();
  auto request = [&](int i) {                              // one thread
    const int s = i % STAGES;
    const float* w = p.work + (static_cast<long>(first + i) * p.H + head) * p.work_stride;
    fi::mbar_expect_tx(&full[s], kStage * 4);
    bulk_load(smem + s * kStage, w, kBase * 4, &full[s]);
    bulk_load(smem + s * kStage + kBase, w + kBase + slice * COLS * 32, COLS * 128, &full[s]);
  };
  int issued = 0;
  if (tid == 0)
    for (; issued < min(STAGES, chunks); ++issued) request(issued);

  // the sequence's convolution inputs that the next portion needs
  {
    const int keep = min(n, p.taps - 1);
    const long per = static_cast<long>(p.C);
    for (long i = static_cast<long>(blockIdx.x) * THREADS + tid; i < keep * per; i += static_cast<long>(gridDim.x) * THREADS) {
      const int back = static_cast<int>(i / per) + 1, ch = static_cast<int>(i % per);
      p.ring[(static_cast<long>(slot) * p.taps + (seq_len - back) % p.taps) * p.C + ch] =
          ld_any(p.qkv, (t_begin + n - back) * p.ld + ch, p.out_type);
    }
  }

  f2 S[NP][CPL];
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int row = range * RPL + 2 * i;
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      float a = 0.f, bb = 0.f;
      if (!fresh && col0 + c < p.dv) {
        if (row < p.d) a = S0[static_cast<long>(row) * p.dv + col0 + c];
        if (row + 1 < p.d) bb = S0[static_cast<long>(row + 1) * p.dv + col0 + c];
      }
      S[i][c] = pack2(a, bb);
    }
  }
  // partial products of 16 operand rows with this lane's part of S
  auto products = [&](const float* a) {
    float* out = part + range * 16 * COLS + lcol;
#pragma unroll 4
    for (int row = 0; row < 16; ++row) {
      f2 acc[CPL][2];
#pragma unroll
      for (int q = 0; q < NP; q += 2) {
        const float4 v = *reinterpret_cast<const float4*>(a + row * DP + q * 2);
        const f2 v0 = pack2(v.x, v.y), v1 = pack2(v.z, v.w);
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          acc[c][0] = q == 0 ? mul2(v0, S[0][c]) : fma2(v0, S[q][c], acc[c][0]);
          acc[c][1] = q == 0 ? mul2(v1, S[1][c]) : fma2(v1, S[q + 1][c], acc[c][1]);
        }
      }
      float y[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        float x0, x1, x2, x3;
        unpack2(acc[c][0], x0, x1);
        unpack2(acc[c][1], x2, x3);
        y[c] = (x0 + x1) + (x2 + x3);
      }
      if constexpr (CPL == 2) *reinterpret_cast<float2*>(out + row * COLS) = make_float2(y[0], y[CPL - 1]);
      else out[row * COLS] = y[0];
    }
  };
  // four columns of one row: the start value plus the row ranges' partial products
  auto gather = [&](const float* base, int row, int c4) {
    float4 y = *reinterpret_cast<const float4*>(base + (c4 >> 2) * 512 + row * 16 + (c4 & 3) * 4);
#pragma unroll
    for (int r = 0; r < PARTS; ++r) {
      const float4 x = *reinterpret_cast<const float4*>(part + (r * 16 + row) * COLS + c4 * 4);
      y.x += x.x; y.y += x.y; y.z += x.z; y.w += x.w;
    }
    return y;
  };
  constexpr int kGroups = COLS / 4;                        // groups of four columns per row
  bool ok = true;
  int waited = chunks;
  for (int i = 0; i < chunks; ++i) {
    const int s = i % STAGES;
    if (!fi::mbar_wait(&full[s], (i / STAGES) & 1)) {
      fi::set_status(status, fi::kStatusTimeoutFull);
      ok = false;
    }
    // the meeting also frees the stage and the partial sums of the chunk before (and tells everybody about a wait that
    // ran out)
    if (__syncthreads_or(ok ? 0 : 1)) { ok = false; waited = i; break; }
    if (STAGES > 1 && i > 0 && tid == 0 && issued < chunks) request(issued++);
    const float* st = smem + s * kStage;
    const float* base = st + kBase;
    products(st + range * RPL);                            // -W S
    __syncthreads();
    for (int g = tid; g < 16 * kGroups; g += THREADS)
      *reinterpret_cast<float4*>(su + g * 4) = gather(base, g / kGroups, g % kGroups);
    __syncthreads();
    products(st + 16 * DP + range * RPL);                  // Q S
    // S <- E_16 S + sum_j (E_16 / E_j) k_j u_j^T
#pragma unroll
    for (int q = 0; q < NP; q += 2) {
      const float4 v = *reinterpret_cast<const float4*>(st + 48 * DP + range * RPL + q * 2);
      const f2 v0 = pack2(v.x, v.y), v1 = pack2(v.z, v.w);
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        S[q][c] = mul2(v0, S[q][c]);
        S[q + 1][c] = mul2(v1, S[q + 1][c]);
      }
    }
#pragma unroll 4
    for (int j = 0; j < 16; ++j) {
      f2 uu[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        const float x = su[j * COLS + lcol + c];
        uu[c] = pack2(x, x);
      }
      const float* k = st + (32 + j) * DP + range * RPL;
#pragma unroll
      for (int q = 0; q < NP; q += 2) {
        const float4 v = *reinterpret_cast<const float4*>(k + q * 2);
        const f2 v0 = pack2(v.x, v.y), v1 = pack2(v.z, v.w);
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          S[q][c] = fma2(v0, uu[c], S[q][c]);
          S[q + 1][c] = fma2(v1, uu[c], S[q + 1][c]);
        }
      }
    }
    __syncthreads();
    for (int g = tid; g < 16 * kGroups; g += THREADS) {
      const int row = g / kGroups, c4 = g % kGroups, tok = i * kTok + row, col = slice * COLS + c4 * 4;
      if (tok >= n || col >= p.dv) continue;
      const float4 y = gather(base + 256, row, c4);
      float* dst = p.o + (static_cast<long>(t_begin + tok) * p.H + head) * p.dv + col;
      if (p.vec_o) {
        *reinterpret_cast<float4*>(dst) = y;
      } else {
        const float o[4] = {y.x, y.y, y.z, y.w};
        for (int c = 0; c < 4 && col + c < p.dv; ++c) dst[c] = o[c];
      }
    }
    if constexpr (STAGES == 1) {                           // the only stage has to be read to the end first
      __syncthreads();
      if (tid == 0 && issued < chunks) request(issued++);
    }
  }
  if (!ok) {                                               // uniform: leave once the copies in flight have landed
    if (tid == 0)
      for (int i = waited; i < issued; ++i) fi::mbar_wait(&full[i % STAGES], (i / STAGES) & 1);
    return;
  }
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int row = range * RPL + 2 * i;
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      float a, bb;
      unpack2(S[i][c], a, bb);
      if (col0 + c < p.dv) {
        if (row < p.d) S0[static_cast<long>(row) * p.dv + col0 + c] = a;
        if (row + 1 < p.d) S0[static_cast<long>(row + 1) * p.dv + col0 + c] = bb;
      }
    }
  }
}

// One token per sequence.  Block: one (head, sequence); thread: VEC columns of every RY-th row.  STAGED: the state waits in
// shared memory between the two passes over it (every thread copies, and reads back, its own part); else it is read twice.
template <int VEC, bool STAGED, typename T>
__global__ void __launch_bounds__(256) delta_step_kernel(const DeltaParams p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  extern __shared__ __align__(128) float smem[];
  __shared__ float red[2][8];
  const int head = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int len = p.seq_lens[b], slot = p.slots[b];
  const int d = p.d, dv = p.dv, taps = p.taps;
  const long orow = static_cast<long>(b) * p.H * dv + static_cast<long>(head) * dv;
  if (len <= 0 || slot < 0 || slot >= p.num_slots) {       // padded row of a decode bucket
    for (int j = tid; j < dv; j += 256) st_any(p.out, orow + j, p.out_type, 0.f);
    return;
  }
  const int nx = (dv + VEC - 1) / VEC;                     // threads across the columns (<= 256)
  const int ry_n = 256 / nx;
  const int cx = tid % nx, ry = tid / nx;
  const bool fresh = len == 1;
  float* S = p.pool + (static_cast<long>(slot) * p.H + head) * d * dv;
  const float* old = STAGED ? smem : S;
  if constexpr (STAGED) {                                  // in flight while the operands are prepared
    if (!fresh && ry < ry_n)
      for (int r = ry; r < d; r += ry_n)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(fi::smem_u32(smem + r * dv + cx * VEC)),
                     "l"(S + static_cast<long>(r) * dv + cx * VEC)
                     : "memory");
  }
  auto fetch = [&](int r, float* s) {
    const float* row = old + static_cast<long>(r) * dv + cx * VEC;
    if constexpr (VEC == 4) {
      const float4 x = *reinterpret_cast<const float4*>(row);
      s[0] = x.x; s[1] = x.y; s[2] = x.z; s[3] = x.w;
    } else {
      s[0] = row[0];
    }
  };
  float* sq = smem + (STAGED ? static_cast<long>(d) * dv : 0);   // [d]
  float* sk = sq + d;               // [d]
  float* sg = sk + d;               // [d]
  float* sv = sg + d;               // [dv]
  float* so = sv + dv;              // [ry][dv] partial sums
  const int pos = len - 1, group = p.H / p.G, kvh = head / group;
  const int cq = kvh * d, ck = p.G * d + kvh * d, cv = 2 * p.G * d + head * dv;
  float* ring = p.ring + static_cast<long>(slot) * taps * p.C;
  const T* x = reinterpret_cast<const T*>(p.qkv) + b * p.ld;
  float ssq = 0.f, ssk = 0.f;
  for (int c = tid; c < 2 * d + dv; c += 256) {
    const int ch = c < d ? cq + c : (c < 2 * d ? ck + c - d : cv + c - 2 * d);
    const float* w = p.conv + static_cast<long>(ch) * taps;
    const float now = to_f(x[ch]);
    float y = w[taps - 1] * now;
    for (int j = 1; j < taps; ++j)
      if (pos - j >= 0) y = fmaf(w[taps - 1 - j], ring[((pos - j) % taps) * p.C + ch], y);
    if (c >= 2 * d || head % group == 0) ring[(pos % taps) * p.C + ch] = now;
    y *= sigmoidf(y);
    if (c < d) { sq[c] = y; ssq += y * y; }
    else if (c < 2 * d) { sk[c - d] = y; ssk += y * y; }
    else sv[c - 2 * d] = y;
  }
  const float rate = p.rate[head];
  for (int c = tid; c < d; c += 256) sg[c] = decay_exp(-rate * softplusf(p.z[b * p.ldz + head * d + c] + p.bias[head * d + c]));
  const float beta = sigmoidf(p.b[b * p.ldb + head]);
  for (int m = 16; m > 0; m >>= 1) {
    ssq += __shfl_xor_sync(0xffffffffu, ssq, m);
    ssk += __shfl_xor_sync(0xffffffffu, ssk, m);
  }
  if ((tid & 31) == 0) { red[0][tid >> 5] = ssq; red[1][tid >> 5] = ssk; }
  __syncthreads();
  ssq = ssk = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) { ssq += red[0][w]; ssk += red[1][w]; }
  const float fq = p.q_scale / sqrtf(ssq + kUnitEps), fk = 1.f / sqrtf(ssk + kUnitEps);
  // first pass: S^T k of the decayed state
  float acc[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
  if (ry < ry_n) {
    if (!fresh) {
      if constexpr (STAGED) asm volatile("cp.async.wait_all;" ::: "memory");
#pragma unroll 4
      for (int r = ry; r < d; r += ry_n) {
        float s[VEC];
        fetch(r, s);
        const float gk = sg[r] * sk[r];
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = fmaf(gk, s[e], acc[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e)
      if (cx * VEC + e < dv) so[ry * dv + cx * VEC + e] = acc[e];
  }
  __syncthreads();
  float u[VEC], o[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) { u[e] = 0.f; o[e] = 0.f; }
  if (ry < ry_n) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      const int c = cx * VEC + e;
      float a = 0.f;
      for (int r = 0; r < ry_n; ++r) a += so[r * dv + c];
      u[e] = beta * (sv[c] - fk * a);
    }
  }
  __syncthreads();
  // second pass: the write, the read-out and the new state
  if (ry < ry_n) {
#pragma unroll 4
    for (int r = ry; r < d; r += ry_n) {
      float s[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) s[e] = 0.f;
      if (!fresh) fetch(r, s);
      const float k = fk * sk[r], q = sq[r], g = sg[r];
      float* row = S + static_cast<long>(r) * dv + cx * VEC;
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        s[e] = fmaf(k, u[e], g * s[e]);
        o[e] = fmaf(q, s[e], o[e]);
      }
      if constexpr (VEC == 4) *reinterpret_cast<float4*>(row) = make_float4(s[0], s[1], s[2], s[3]);
      else row[0] = s[0];
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) so[ry * dv + cx * VEC + e] = o[e];
  }
  __syncthreads();
  float ss = 0.f;
  for (int j = tid; j < dv; j += 256) {
    float a = 0.f;
    for (int r = 0; r < ry_n; ++r) a += so[r * dv + j];
    a *= fq;
    so[j] = a;                      // row 0 of its own column: nobody else reads it any more
    ss += a * a;
  }
  for (int m = 16; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  if ((tid & 31) == 0) red[0][tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) tot += red[0][w];
  const float inv = 1.f / sqrtf(tot / static_cast<float>(dv) + p.eps);
  for (int j = tid; j < dv; j += 256) {
    float y = so[j] * inv * p.norm_w[j];
    if (p.gate != nullptr) y *= sigmoidf(ld_any(p.gate, b * p.ldg + head * dv + j, p.gate_type));
    st_any(p.out, orow + j, p.out_type, y);
  }
}

int check(const DeltaParams& p, int type) {
  if (p.B <= 0 || p.H <= 0 || p.G <= 0 || p.H % p.G != 0 || p.d <= 0 || p.dv <= 0 || p.taps < 1 || p.taps > 16 ||
      p.B > 65535 || p.H > 65535 || type < 0 || type > 2 || p.num_slots <= 0)
    return -10;
  return 0;
}

template <int DP, int LR, int CPL>
int launch_scan(const DeltaParams& p, int* status, cudaStream_t s) {
  constexpr int WARPS = DP <= 256 ? 8 : 16, RPL = DP / (WARPS * LR), COLS = 32 / LR * CPL;
  constexpr int STAGES = DP <= 256 ? 2 : 1;
  constexpr int smem = (STAGES * (49 * DP + 32 * COLS) + WARPS * LR * 16 * COLS + 16 * COLS) * 4;
  auto kern = delta_scan_kernel<RPL, LR, CPL, WARPS, STAGES>;
  cudaError_t e = fi::ensure_dynamic_smem(kern, smem);
  if (e != cudaSuccess) return static_cast<int>(e);
  return static_cast<int>(fi::launch_kernel(kern, dim3(p.H * (p.dvp / COLS), p.B), dim3(WARPS * 32), smem, s, 0, p, status));
}

template <int DP>
int pick_cols(const DeltaParams& p, int* status, cudaStream_t s) {
  // wide tiles read every operand row the fewest times, narrow ones fill the device when there are few sequences
  const long ctas = static_cast<long>(p.B) * p.H * (p.dvp / 64);
  if constexpr (DP <= 256) {
    if (ctas >= 120) return launch_scan<DP, 1, 2>(p, status, s);
    if (ctas >= 60) return launch_scan<DP, 1, 1>(p, status, s);
  }
  return launch_scan<DP, 2, 1>(p, status, s);
}

template <typename T>
cudaError_t launch_chunks(const DeltaParams& p, int smem, cudaStream_t s) {
  auto go = [&](auto kern) {
    const cudaError_t e = fi::ensure_dynamic_smem(kern, smem);
    return e != cudaSuccess ? e : fi::launch_kernel(kern, dim3(p.n_chunks, p.H), dim3(256), smem, s, 0, p);
  };
  if (p.taps == 4) return go(delta_chunk_kernel<T, 4>);
  if (p.taps == 3) return go(delta_chunk_kernel<T, 3>);
  if (p.taps == 2) return go(delta_chunk_kernel<T, 2>);
  return go(delta_chunk_kernel<T, 0>);
}

}  // namespace

// Floats of the work buffer per (chunk of 16 tokens, head), or -1 for sizes outside the kernels.
extern "C" long fi_delta_work_floats(int d, int dv) {
  if (d <= 0 || dv <= 0 || d > 512) return -1;
  const int dp = d <= 64 ? 64 : d <= 128 ? 128 : d <= 256 ? 256 : 512;
  return work_floats(dp, (dv + 63) / 64 * 64);
}

// Portions of sequences.  qkv: type (0 bf16, 1 fp16, 2 fp32) rows of pitch ld, q (G * d) | k (G * d) | v (H * dv); z, b:
// fp32 rows; conv: fp32 [C, taps]; rate, bias: fp32 [H], [H * d]; pool: fp32 [num_slots, H, d, dv]; ring: fp32
// [num_slots, taps, C]; slots, seq_lens: int32 [B]; cu_q, chunk_base: int32 [B + 1] (chunk_base: running count of
// ceil(portion / 16), n_chunks in total); work: n_chunks * H * fi_delta_work_floats(d, dv) floats, 16-byte aligned;
// o: fp32 [T, H, dv].
extern "C" int fi_delta_portions(const void* qkv, long ld, const float* z, long ldz, const float* b, long ldb,
                                 const float* conv, const float* rate, const float* bias, float* pool, float* ring,
                                 const int* slots, const int* cu_q, const int* seq_lens, const int* chunk_base,
                                 int n_chunks, float* work, float* o, int B, int H, int G, int d, int dv, int taps,
                                 int num_slots, int type, int* status, void* stream) {
  if (B <= 0 || n_chunks <= 0) return 0;
  DeltaParams p = {};
  p.qkv = qkv; p.ld = ld; p.z = z; p.ldz = ldz; p.b = b; p.ldb = ldb; p.conv = conv; p.rate = rate; p.bias = bias;
  p.pool = pool; p.ring = ring; p.slots = slots; p.cu_q = cu_q; p.seq_lens = seq_lens; p.chunk_base = chunk_base;
  p.n_chunks = n_chunks; p.work = work; p.o = o; p.B = B; p.H = H; p.G = G; p.d = d; p.dv = dv; p.taps = taps;
  p.num_slots = num_slots; p.C = 2 * G * d + H * dv; p.q_scale = 1.f / sqrtf(static_cast<float>(d)); p.out_type = type;
  const int bad = check(p, type);
  if (bad != 0) return bad;
  if (d > 512 || (reinterpret_cast<uintptr_t>(work) & 15) != 0) return -11;
  p.dp = d <= 64 ? 64 : d <= 128 ? 128 : d <= 256 ? 256 : 512;
  p.dvp = (dv + 63) / 64 * 64;
  p.work_stride = work_floats(p.dp, p.dvp);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  p.vec_o = dv % 4 == 0 && (reinterpret_cast<uintptr_t>(o) & 15) == 0;
  const long floats = static_cast<long>(kTok) * (5 * ((d + 3) & ~3) + dv) + 560;
  if (floats * 4 > 227 * 1024) return -11;
  const int smem = static_cast<int>(floats * 4);
  const cudaError_t e = type == 0   ? launch_chunks<__nv_bfloat16>(p, smem, s)
                        : type == 1 ? launch_chunks<__half>(p, smem, s)
                                    : launch_chunks<float>(p, smem, s);
  if (e != cudaSuccess) return static_cast<int>(e);
  if (p.dp == 64) return pick_cols<64>(p, status, s);
  if (p.dp == 128) return pick_cols<128>(p, status, s);
  if (p.dp == 256) return pick_cols<256>(p, status, s);
  return pick_cols<512>(p, status, s);
}

// One token per sequence with head norm and output gate.  Operands as above; norm_w: fp32 [dv]; gate: rows of pitch ldg
// of gate_type, or null; out: [B, H * dv] of out_type.  Rows with seq_lens <= 0 are padding: zero output, no state or
// ring row touched.
extern "C" int fi_delta_step(const void* qkv, long ld, const float* z, long ldz, const float* b, long ldb,
                             const float* conv, const float* rate, const float* bias, float* pool, float* ring,
                             const int* slots, const int* seq_lens, const float* norm_w, float eps, const void* gate,
                             long ldg, int gate_type, void* out, int B, int H, int G, int d, int dv, int taps,
                             int num_slots, int type, int out_type, void* stream) {
  if (B <= 0) return 0;
  DeltaParams p = {};
  p.qkv = qkv; p.ld = ld; p.z = z; p.ldz = ldz; p.b = b; p.ldb = ldb; p.conv = conv; p.rate = rate; p.bias = bias;
  p.pool = pool; p.ring = ring; p.slots = slots; p.seq_lens = seq_lens; p.norm_w = norm_w; p.eps = eps; p.gate = gate;
  p.ldg = ldg; p.gate_type = gate_type; p.out = out; p.B = B; p.H = H; p.G = G; p.d = d; p.dv = dv; p.taps = taps;
  p.num_slots = num_slots; p.C = 2 * G * d + H * dv; p.q_scale = 1.f / sqrtf(static_cast<float>(d)); p.out_type = out_type;
  const int bad = check(p, type);
  if (bad != 0) return bad;
  if (gate_type < 0 || gate_type > 2 || out_type < 0 || out_type > 2) return -10;
  const bool vec4 = dv % 4 == 0 && (reinterpret_cast<uintptr_t>(pool) & 15) == 0;
  const int nx = vec4 ? dv / 4 : dv;
  if (nx > 256) return -11;
  const int ry = 256 / nx;
  const long small = (3l * d + dv + static_cast<long>(ry) * dv) * 4, tile = static_cast<long>(d) * dv * 4;
  if (small > 100 * 1024) return -11;
  const bool staged = vec4 && small + tile <= 200 * 1024;
  const int smem = static_cast<int>(staged ? small + tile : small);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define FI_STEP(V, K, TT)                                                                                    \
  {                                                                                                          \
    const cudaError_t e = fi::ensure_dynamic_smem(delta_step_kernel<V, K, TT>, smem);                        \
    if (e != cudaSuccess) return static_cast<int>(e);                                                        \
    return static_cast<int>(fi::launch_kernel(delta_step_kernel<V, K, TT>, dim3(H, B), dim3(256), smem, s, 0, p)); \
  }
#define FI_STEP_T(V, K)                          \
  {                                              \
    if (type == 0) FI_STEP(V, K, __nv_bfloat16)  \
    if (type == 1) FI_STEP(V, K, __half)         \
    FI_STEP(V, K, float)                         \
  }
  if (!vec4) FI_STEP_T(1, false)
  if (!staged) FI_STEP_T(4, false)
  FI_STEP_T(4, true)
#undef FI_STEP_T
#undef FI_STEP
}
