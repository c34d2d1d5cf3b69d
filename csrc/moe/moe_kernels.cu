// Mixture-of-experts support kernels for sm_100a: router top-k, expert alignment (counting sort +
// tile table for the grouped GEMM), activation gather and weighted combine.
//
//   fi_moe_route   : scores -> top-k experts and weights per token, three scoring rules:
//                    0 softmax over all experts, top-k, renormalise (Gemma4: vllm/model_executor/
//                      models/gemma4/moe.py:98-125, optional per-expert scale); selection by score +
//                      correction bias where there is one,
//                    1 sigmoid scores, selection by score + correction bias, weights = normalised
//                      scores x routed scaling (DeepSeek-V3 style),
//                    2 sqrt(softplus) scores with bias (DeepSeek-V4-Flash: deepseek_v4_flash/
//                      gpu_layers.py:323-352).
//                    Optionally the experts form equal groups of neighbours and only the best groups (by their
//                    largest selection score, or the sum of their two largest) can be chosen.
//   fi_moe_align   : counting sort of the (token, k) routes by expert restricted to the experts this
//                    rank owns; emits sorted route ids, the inverse map, per-expert offsets and the
//                    tile table (expert, first row, rows) consumed by fi_awq_gemm_grouped.
//   fi_moe_gather  : x_sorted[slot] = x[route / k]
//   fi_moe_combine : out[t] = sum_k w[t,k] * y_sorted[slot(t,k)]  (+ optional residual), fp32 sums in
//                    a fixed order, so the result does not depend on the order of the sort.
//   fi_moe_expert_rows : expert products on the general cores in 32-bit arithmetic (32-bit models, odd sizes)
// The reference routes with torch.topk/softmax and runs experts in Python loops or M<=16 Triton
// kernels (vllm/kernels/triton/gemma4_moe_int4.py); nothing there sorts tokens by expert on device.
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <math_constants.h>
#include <stdint.h>

#include "../common/launch.cuh"
#include "../common/ptx.cuh"
#include "../gemm/comm_desc.h"

namespace {

constexpr int kMaxExpertsPerLane = 16;   // experts <= 512

// Order-preserving map of scores to unsigned numbers above 0; what is no number (and whatever is out of the race) is 0.
__device__ __forceinline__ unsigned score_key(float v) {
  const unsigned u = __float_as_uint(v);
  if ((u & 0x7fffffffu) > 0x7f800000u) return 0u;
  return u ^ ((u >> 31) ? 0xffffffffu : 0x80000000u);
}
__device__ __forceinline__ float key_score(unsigned k) {
  return __uint_as_float(k ^ ((k >> 31) ? 0x80000000u : 0xffffffffu));
}

// One warp per token; lane l owns experts l, l + 32, ... (PER of them, in registers).
template <int PER>
__global__ void moe_route_kernel(const float* __restrict__ logits, const float* __restrict__ bias,
                                 const float* __restrict__ expert_scale, int* __restrict__ topk_ids,
                                 float* __restrict__ topk_w, long ld, int T, int E, int K, int mode,
                                 int renorm, float routed_scale, int groups, int keep_groups, int group_best) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  constexpr unsigned kAll = 0xffffffffu;
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (t >= T) return;
  const float* row = logits + t * ld;
  float score[PER];     // value used for the weight
  unsigned key[PER];    // value used for the selection
  float mx = -CUDART_INF_F;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = i * 32 + lane;
    score[i] = e < E ? row[e] : -CUDART_INF_F;
    mx = fmaxf(mx, score[i]);
  }
  if (mode == 0) {
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(kAll, mx, o));
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      score[i] = i * 32 + lane < E ? __expf(score[i] - mx) : 0.f;
      sum += score[i];
    }
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(kAll, sum, o);
#pragma unroll
    for (int i = 0; i < PER; ++i) score[i] /= sum;
  } else {
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const float x = score[i];
      score[i] = mode == 1 ? 1.f / (1.f + __expf(-x)) : sqrtf(x > 20.f ? x : log1pf(__expf(x)));
    }
  }
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = i * 32 + lane;
    key[i] = e < E ? score_key(score[i] + (bias ? bias[e] : 0.f)) : 0u;
  }
  // the largest key among this warp's entries that `open` lets through and the lowest expert that has it
  auto best_of = [&](auto open, int& expert) -> unsigned {
    unsigned b = 0u;
    int at = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (key[i] > b && open(i)) { b = key[i]; at = i * 32 + lane; }
    const unsigned top = __reduce_max_sync(kAll, b);
    expert = static_cast<int>(__reduce_min_sync(kAll, b == top ? static_cast<unsigned>(at) : 0x7fffffffu));
    return top;
  };
  if (keep_groups < groups) {
    // kept groups are bits in registers: bit g & 31 of word g >> 5; ties go to the lower group
    const int size = E / groups;
    unsigned kept[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) kept[i] = 0u;
    auto is_kept = [&](int g) {
      bool in = false;
#pragma unroll
      for (int w = 0; w < PER; ++w) in |= w == (g >> 5) && ((kept[w] >> (g & 31)) & 1u);
      return in;
    };
    auto keep = [&](int g) {
#pragma unroll
      for (int w = 0; w < PER; ++w)
        if (w == (g >> 5)) kept[w] |= 1u << (g & 31);
    };
    int group[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) group[i] = (i * 32 + lane) / size;
    if (group_best < 2) {
      // the best group left is the one of the best expert left
      for (int k = 0; k < keep_groups; ++k) {
        int e;
        if (best_of([&](int i) { return !is_kept(group[i]); }, e) != 0u) keep(e / size);
      }
    } else {
      float gscore[PER];                                       // score of group g ends in lane g % 32
#pragma unroll
      for (int i = 0; i < PER; ++i) gscore[i] = -CUDART_INF_F;
      for (int g = 0; g < groups; ++g) {
        float m1 = -CUDART_INF_F, m2 = -CUDART_INF_F;          // the two largest of this lane's experts in the group
#pragma unroll
        for (int i = 0; i < PER; ++i) {
          if (group[i] == g && key[i] != 0u) {
            const float v = key_score(key[i]);
            m2 = fmaxf(m2, fminf(m1, v));
            m1 = fmaxf(m1, v);
          }
        }
        for (int o = 16; o > 0; o >>= 1) {
          const float o1 = __shfl_xor_sync(kAll, m1, o), o2 = __shfl_xor_sync(kAll, m2, o);
          m2 = fmaxf(fmaxf(m2, o2), fminf(m1, o1));
          m1 = fmaxf(m1, o1);
        }
#pragma unroll
        for (int w = 0; w < PER; ++w)
          if (g == w * 32 + lane) gscore[w] = size > 1 ? m1 + m2 : m1;
      }
      for (int k = 0; k < keep_groups; ++k) {
        unsigned b = 0u;
        int at = 0x7fffffff;
#pragma unroll
        for (int w = 0; w < PER; ++w) {
          const int g = w * 32 + lane;
          const unsigned v = g < groups && !((kept[w] >> lane) & 1u) ? score_key(gscore[w]) : 0u;
          if (v > b) { b = v; at = g; }
        }
        const unsigned top = __reduce_max_sync(kAll, b);
        const int g = static_cast<int>(__reduce_min_sync(kAll, b == top ? static_cast<unsigned>(at) : 0x7fffffffu));
        if (top != 0u) keep(g);
      }
    }
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (!is_kept(group[i])) key[i] = 0u;
  }
  float wsum = 0.f;
  float my_w = 0.f;
  int my_id = 0;
  for (int k = 0; k < K; ++k) {
    int bi;
    if (best_of([](int) { return true; }, bi) == 0u) bi = 0;  // no comparable score left (a router output that is no number)
    // the owner lane reads the weight score and retires the expert
    float w = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (i * 32 + lane == bi) { w = score[i]; key[i] = 0u; }
    w = __shfl_sync(kAll, w, bi & 31);
    wsum += w;
    if (lane == k) { my_w = w; my_id = bi; }
  }
  if (lane < K) {
    float w = my_w;
    if (renorm) w = w / fmaxf(wsum, 1e-20f);
    w *= routed_scale;
    if (expert_scale != nullptr) w *= expert_scale[my_id];
    topk_ids[static_cast<long>(t) * K + lane] = my_id;
    topk_w[static_cast<long>(t) * K + lane] = w;
  }
}

// One CTA.  Routes to experts outside [e_lo, e_hi) are dropped (slot_of = -1).
// Expert of route i: topk_ids[i], or (assigned) row ids[i / top] of a table [vocab, top].
struct RouteIds {
  const int* topk_ids;
  const int* table;
  const long long* ids;
  int vocab, top;
  __device__ __forceinline__ int operator[](int i) const {
    if (table == nullptr) return topk_ids[i];
    const int t = i / top;
    const long long id = ids[t];
    return table[(id < 0 || id >= vocab ? 0 : id) * top + i - t * top];      // padded rows of a decode bucket carry stale ids
  }
};

__global__ void moe_align_kernel(const RouteIds routes, int n_routes, int e_lo, int e_hi,
                                 int bn, int* __restrict__ sorted_route, int* __restrict__ slot_of,
                                 int* __restrict__ expert_offsets, int* __restrict__ tile_expert,
                                 int* __restrict__ tile_row0, int* __restrict__ tile_rows,
                                 int* __restrict__ n_tiles) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  extern __shared__ int sm[];
  const int EL = e_hi - e_lo;
  int* counts = sm;            // [EL]
  int* offs = sm + EL;         // [EL + 1]
  int* cursor = offs + EL + 1; // [EL]
  for (int i = threadIdx.x; i < EL; i += blockDim.x) { counts[i] = 0; cursor[i] = 0; }
  __syncthreads();
  for (int i = threadIdx.x; i < n_routes; i += blockDim.x) {
    const int e = routes[i];
    if (e >= e_lo && e < e_hi) atomicAdd(&counts[e - e_lo], 1);
  }
  __syncthreads();
  if (threadIdx.x < 32) {
    // one warp: every lane owns a contiguous range of experts, the ranges are chained by a warp prefix sum
    const int lane = threadIdx.x;
    const int per = (EL + 31) / 32;
    const int e0 = min(EL, lane * per), e1 = min(EL, e0 + per);
    int rows = 0, tiles = 0;
    for (int e = e0; e < e1; ++e) { rows += counts[e]; tiles += (counts[e] + bn - 1) / bn; }
    int row_pre = rows, tile_pre = tiles;
    for (int o = 1; o < 32; o <<= 1) {
      const int r = __shfl_up_sync(0xffffffffu, row_pre, o), t = __shfl_up_sync(0xffffffffu, tile_pre, o);
      if (lane >= o) { row_pre += r; tile_pre += t; }
    }
    int acc = row_pre - rows, nt = tile_pre - tiles;
    for (int e = e0; e < e1; ++e) {
      offs[e] = acc;
      for (int r = 0; r < counts[e]; r += bn) {
        tile_expert[nt] = e;
        tile_row0[nt] = acc + r;
        tile_rows[nt] = min(bn, counts[e] - r);
        ++nt;
      }
      acc += counts[e];
    }
    if (lane == 31) {
      offs[EL] = row_pre;
      *n_tiles = tile_pre;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i <= EL; i += blockDim.x) expert_offsets[i] = offs[i];
  for (int i = threadIdx.x; i < n_routes; i += blockDim.x) {
    const int e = routes[i];
    if (e >= e_lo && e < e_hi) {
      const int slot = offs[e - e_lo] + atomicAdd(&cursor[e - e_lo], 1);
      sorted_route[slot] = i;
      slot_of[i] = slot;
    } else {
      slot_of[i] = -1;
    }
  }
}

// Tile table of E stacked matrices of T rows each.
__global__ void __launch_bounds__(256) stack_tiles_kernel(int E, int T, int bn, int per, int* __restrict__ tile_expert,
                                                          int* __restrict__ tile_row0, int* __restrict__ tile_rows,
                                                          int* __restrict__ n_tiles) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i == 0) *n_tiles = E * per;
  if (i >= E * per) return;
  const int e = i / per, r = (i % per) * bn;
  tile_expert[i] = e;
  tile_row0[i] = e * T + r;
  tile_rows[i] = min(bn, T - r);
}

template <typename T>
__global__ void moe_gather_kernel(const T* __restrict__ x, const int* __restrict__ sorted_route,
                                  const int* __restrict__ expert_offsets, int EL, int K, int H,
                                  T* __restrict__ x_sorted) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  const int slot = blockIdx.x;
  if (slot >= expert_offsets[EL]) return;
  const int tok = sorted_route[slot] / K;
  const uint4* src = reinterpret_cast<const uint4*>(x + static_cast<long>(tok) * H);
  uint4* dst = reinterpret_cast<uint4*>(x_sorted + static_cast<long>(slot) * H);
  for (int i = threadIdx.x; i < H / 8; i += blockDim.x) dst[i] = src[i];
}

template <typename T>
__global__ void moe_combine_kernel(const T* __restrict__ y_sorted, const int* __restrict__ slot_of,
                                   const float* __restrict__ topk_w, const T* __restrict__ residual,
                                   T* __restrict__ out, int K, int H) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  const int t = blockIdx.x;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < H / 8; c += blockDim.x * gridDim.y) {
    float acc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = 0.f;
    for (int k = 0; k < K; ++k) {
      // a null map means the rows are already in (token, k) order
      const int slot = slot_of ? slot_of[static_cast<long>(t) * K + k] : t * K + k;
      if (slot < 0) continue;
      const float w = topk_w[static_cast<long>(t) * K + k];
      uint4 raw = *reinterpret_cast<const uint4*>(y_sorted + static_cast<long>(slot) * H + c * 8);
      const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] += w * static_cast<float>(e[j]);
    }
    if (residual != nullptr) {
      uint4 raw = *reinterpret_cast<const uint4*>(residual + static_cast<long>(t) * H + c * 8);
      const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] += static_cast<float>(e[j]);
    }
    uint4 o;
    T* oe = reinterpret_cast<T*>(&o);
#pragma unroll
    for (int j = 0; j < 8; ++j) oe[j] = static_cast<T>(acc[j]);
    *reinterpret_cast<uint4*>(out + static_cast<long>(t) * H + c * 8) = o;
  }
}

// Expert-parallel combine fused with the all-reduce: every rank sums the routed outputs of ITS
// experts for a token, pushes that fp32 partial straight into every peer's receive slab over NVLink
// (each 8-byte word = one value + the call's epoch, so the receiver needs neither a fence nor a
// separate flag), then adds the peers' partials in rank order (bitwise identical on all ranks) plus
// the residual and writes the token.  One CTA per token; waits are bounded.
struct CombineComm {
  int world, rank;
  long slab_elems;                  // values per (parity, source rank) slab
  unsigned long long recv[8];       // low-latency receive area of rank d, as mapped here
  unsigned int* epoch;              // local: completed fused calls
  unsigned int* done;               // local: finished CTAs of this call
  int* status;
  int phases;
};

template <typename T>
__global__ void moe_combine_allreduce_kernel(const T* __restrict__ y_sorted, const int* __restrict__ slot_of,
                                             const float* __restrict__ topk_w, const T* __restrict__ residual,
                                             T* __restrict__ out, int K, int H, const CombineComm c) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  __shared__ volatile int aborted;
  if (threadIdx.x == 0) aborted = 0;
  __syncthreads();
  const unsigned int epoch_now = *c.epoch + 1u;
  const long parity = epoch_now & 1u;
  const int t = blockIdx.x;
  const int phases = c.phases != 0 ? c.phases : 3;   // 1 = push partials, 2 = sum + store (split only when one GPU emulates several ranks)
  for (int ch = threadIdx.x; ch < H / 8; ch += blockDim.x) {
    float acc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = 0.f;
    for (int k = 0; k < K; ++k) {
      const int slot = slot_of ? slot_of[static_cast<long>(t) * K + k] : t * K + k;
      if (slot < 0) continue;   // routed to an expert of another rank
      const float w = topk_w[static_cast<long>(t) * K + k];
      uint4 raw = *reinterpret_cast<const uint4*>(y_sorted + static_cast<long>(slot) * H + ch * 8);
      const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] += w * static_cast<float>(e[j]);
    }
    const long elem = static_cast<long>(t) * H + ch * 8;
    const long my_off = (parity * c.world + c.rank) * c.slab_elems + elem;
    for (int d = 0; d < c.world; ++d) {
      if (d == c.rank || !(phases & 1)) continue;
      uint4* dst = reinterpret_cast<uint4*>(c.recv[d]) + (my_off >> 1);
#pragma unroll
      for (int q = 0; q < 4; ++q)
        fi::st_volatile_v4(dst + q, make_uint4(__float_as_uint(acc[2 * q]), epoch_now,
                                               __float_as_uint(acc[2 * q + 1]), epoch_now));
    }
    if (!(phases & 2)) continue;
    float sum[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) sum[j] = 0.f;
    for (int s = 0; s < c.world; ++s) {
      float v[8];
      if (s == c.rank) {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = acc[j];
      } else {
        const long off = (parity * c.world + s) * c.slab_elems + elem;
        const uint4* src = reinterpret_cast<const uint4*>(c.recv[c.rank]) + (off >> 1);
        const long long w0 = clock64();
        uint4 wv[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) wv[q] = fi::ld_volatile_v4(src + q);   // four independent loads in flight
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          while (wv[q].y != epoch_now || wv[q].w != epoch_now) {
            if (aborted || clock64() - w0 > FI_WAIT_CYCLES) {
              fi::set_status(c.status, fi::kStatusTimeoutPeer);
              aborted = 1;
              break;
            }
            wv[q] = fi::ld_volatile_v4(src + q);
          }
          v[2 * q] = __uint_as_float(wv[q].x);
          v[2 * q + 1] = __uint_as_float(wv[q].z);
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) sum[j] += v[j];
    }
    if (residual != nullptr) {
      uint4 raw = *reinterpret_cast<const uint4*>(residual + elem);
      const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
      for (int j = 0; j < 8; ++j) sum[j] += static_cast<float>(e[j]);
    }
    if (!aborted) {
      uint4 o;
      T* oe = reinterpret_cast<T*>(&o);
#pragma unroll
      for (int j = 0; j < 8; ++j) oe[j] = static_cast<T>(sum[j]);
      *reinterpret_cast<uint4*>(out + elem) = o;
    }
  }
  // the last CTA of the call publishes the new epoch for the next fused call
  if (!(phases & 2)) return;
  __syncthreads();
  if (threadIdx.x == 0) {
    __threadfence();
    if (atomicAdd(c.done, 1u) == gridDim.x - 1) {
      *c.done = 0;
      __threadfence();
      *reinterpret_cast<volatile unsigned int*>(c.epoch) = epoch_now;
    }
  }
}

// Expert products on the general cores: 32 rows x 64 outputs per block, 32-bit arithmetic.
//   gather: out[row] = act(Wg x) * (Wu x), or its clipped form (act 4), with x = X[sorted_route[row] / top] and weights [Wg (N rows); Wu (N rows)]
//   else:   out[row] = W x with x = X[row]
struct ExpertRows {
  const void* x;            // rows of pitch ldx
  const void* w;            // [experts, gather ? 2 N : N, K]
  void* out;                // rows of pitch ldo
  const int* sorted_route;
  const int* tile_expert;
  const int* tile_row0;
  const int* tile_rows;     // at most 32
  const int* n_tiles;
  long ldx, ldo;
  int N, K, top, gather, act;
  float limit;
};

template <typename T>
__global__ void __launch_bounds__(256) moe_expert_rows_kernel(const ExpertRows p) {
  fi::pdl_launch_dependents();
  fi::pdl_wait();
  constexpr int RB = 32, NB = 64, KB = 32;
  const int tile = blockIdx.y;
  if (tile >= *p.n_tiles) return;
  const int e = p.tile_expert[tile], row0 = p.tile_row0[tile], rows = min(p.tile_rows[tile], RB);
  const int n0 = blockIdx.x * NB;
  __shared__ float sx[KB][RB + 1], swg[KB][NB + 1], swu[KB][NB + 1];
  __shared__ long src[RB];
  const int tid = threadIdx.x;
  if (tid < RB) src[tid] = tid < rows ? static_cast<long>(p.gather ? p.sorted_route[row0 + tid] / p.top : row0 + tid) * p.ldx : -1;
  __syncthreads();
  const T* x = reinterpret_cast<const T*>(p.x);
  const T* wg = reinterpret_cast<const T*>(p.w) + static_cast<long>(e) * (p.gather ? 2 : 1) * p.N * p.K;
  const T* wu = wg + static_cast<long>(p.N) * p.K;
  const int tr = tid >> 4, tn = tid & 15;           // rows tr, tr + 16; outputs tn + 16 i
  float ag[2][4] = {}, au[2][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += KB) {
    for (int i = tid; i < RB * KB; i += 256) {
      const int r = i / KB, k = i % KB;
      sx[k][r] = (src[r] >= 0 && k0 + k < p.K) ? static_cast<float>(x[src[r] + k0 + k]) : 0.f;
    }
    for (int i = tid; i < NB * KB; i += 256) {
      const int n = i / KB, k = i % KB;
      const bool in = n0 + n < p.N && k0 + k < p.K;
      const long at = static_cast<long>(n0 + n) * p.K + k0 + k;
      swg[k][n] = in ? static_cast<float>(wg[at]) : 0.f;
      if (p.gather) swu[k][n] = in ? static_cast<float>(wu[at]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < KB; ++k) {
      const float x0 = sx[k][tr], x1 = sx[k][tr + 16];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float g = swg[k][tn + 16 * i];
        ag[0][i] = fmaf(x0, g, ag[0][i]);
        ag[1][i] = fmaf(x1, g, ag[1][i]);
        if (p.gather) {
          const float u = swu[k][tn + 16 * i];
          au[0][i] = fmaf(x0, u, au[0][i]);
          au[1][i] = fmaf(x1, u, au[1][i]);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int r = tr + 16 * h;
    if (r >= rows) continue;
    T* out = reinterpret_cast<T*>(p.out) + (row0 + r) * p.ldo;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int n = n0 + tn + 16 * i;
      if (n >= p.N) continue;
      float v = ag[h][i];
      if (p.gather && p.act == 4) {
        const float g = fminf(v, p.limit);
        v = g / (1.f + __expf(-1.702f * g)) * (fminf(fmaxf(au[h][i], -p.limit), p.limit) + 1.f);
      } else if (p.gather) {
        v = v / (1.f + __expf(-v)) * au[h][i];
      }
      out[n] = static_cast<T>(v);
    }
  }
}

}  // namespace

#define FI_STREAM(s) reinterpret_cast<cudaStream_t>(s)

// comm: the FiComm descriptor of the symmetric heap with recv[] pointing at the low-latency slabs
extern "C" int fi_moe_combine_allreduce(const void* y_sorted, const int* slot_of, const float* topk_w,
                                        const void* residual, void* out, int T, int K, int H, int dtype,
                                        int* status, void* stream, const FiComm* comm) {
  if (T <= 0) return 0;
  if (H % 8 != 0 || comm == nullptr || comm->world < 2 || comm->world > 8) return -10;
  if (static_cast<long>(T) * H > comm->slab_elems) return -11;
  CombineComm c;
  c.world = comm->world; c.rank = comm->rank; c.slab_elems = comm->slab_elems; c.phases = comm->phases;
  for (int d = 0; d < 8; ++d) c.recv[d] = comm->recv[d];
  c.epoch = reinterpret_cast<unsigned int*>(comm->epoch);
  c.done = reinterpret_cast<unsigned int*>(comm->done);
  c.status = status;
  if (dtype == 0)
    fi::launch_kernel(moe_combine_allreduce_kernel<__nv_bfloat16>, dim3(T), dim3(128), 0, FI_STREAM(stream), 0,
                      (const __nv_bfloat16*)y_sorted, slot_of, topk_w, (const __nv_bfloat16*)residual,
                      (__nv_bfloat16*)out, K, H, c);
  else
    fi::launch_kernel(moe_combine_allreduce_kernel<__half>, dim3(T), dim3(128), 0, FI_STREAM(stream), 0,
                      (const __half*)y_sorted, slot_of, topk_w, (const __half*)residual, (__half*)out, K, H, c);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int fi_moe_route(const float* logits, const float* bias, const float* expert_scale,
                            long ld, int* topk_ids, float* topk_w, int T, int E, int K, int mode, int renorm,
                            float routed_scale, int groups, int keep_groups, int group_best, void* stream) {
  if (T <= 0) return 0;
  if (E > 32 * kMaxExpertsPerLane || K > 32 || K > E || groups < 1 || E % groups != 0 || keep_groups < 1 ||
      keep_groups > groups || K > keep_groups * (E / groups) || ld < E || group_best < 1 || group_best > 2)
    return -10;
  auto kern = E <= 32 ? moe_route_kernel<1> : E <= 64 ? moe_route_kernel<2> : E <= 128 ? moe_route_kernel<4>
              : E <= 256 ? moe_route_kernel<8> : moe_route_kernel<kMaxExpertsPerLane>;
  fi::launch_kernel(kern, dim3((T + 3) / 4), dim3(128), 0, FI_STREAM(stream), 0, logits, bias,
                    expert_scale, topk_ids, topk_w, ld, T, E, K, mode, renorm, routed_scale, groups, keep_groups,
                    group_best);
  return static_cast<int>(cudaGetLastError());
}

// Tile table (as of fi_moe_align) of E stacked matrices of T rows: E * ceil(T / bn) tiles.
extern "C" int fi_stack_tiles(int E, int T, int bn, int* tile_expert, int* tile_row0, int* tile_rows, int* n_tiles, void* stream) {
  if (E <= 0 || T <= 0) return 0;
  if (bn <= 0) return -10;
  const int per = (T + bn - 1) / bn;
  return static_cast<int>(fi::launch_kernel(stack_tiles_kernel, dim3((E * per + 255) / 256), dim3(256), 0, FI_STREAM(stream), 0, E, T, bn,
                                            per, tile_expert, tile_row0, tile_rows, n_tiles));
}

static int launch_align(const RouteIds& routes, int n_routes, int e_lo, int e_hi, int bn, int* sorted_route, int* slot_of,
                        int* expert_offsets, int* tile_expert, int* tile_row0, int* tile_rows, int* n_tiles, void* stream) {
  if (n_routes <= 0) return 0;
  const int EL = e_hi - e_lo;
  if (EL <= 0 || EL > 4096) return -10;
  const size_t smem = (3 * EL + 1) * sizeof(int);
  fi::launch_kernel(moe_align_kernel, dim3(1), dim3(1024), smem, FI_STREAM(stream), 0, routes, n_routes,
                    e_lo, e_hi, bn, sorted_route, slot_of, expert_offsets, tile_expert, tile_row0, tile_rows,
                    n_tiles);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int fi_moe_align(const int* topk_ids, int n_routes, int e_lo, int e_hi, int bn,
                            int* sorted_route, int* slot_of, int* expert_offsets, int* tile_expert,
                            int* tile_row0, int* tile_rows, int* n_tiles, void* stream) {
  return launch_align({topk_ids, nullptr, nullptr, 0, 1}, n_routes, e_lo, e_hi, bn, sorted_route, slot_of, expert_offsets, tile_expert,
                      tile_row0, tile_rows, n_tiles, stream);
}

// The same for experts assigned to token ids: route i is choice i % top of token ids[i / top] in table [vocab, top].
extern "C" int fi_moe_align_assigned(const int* table, const long long* ids, int vocab, int top, int n_routes, int e_hi, int bn,
                                     int* sorted_route, int* slot_of, int* expert_offsets, int* tile_expert, int* tile_row0,
                                     int* tile_rows, int* n_tiles, void* stream) {
  if (table == nullptr || ids == nullptr || vocab <= 0 || top <= 0) return -10;
  return launch_align({nullptr, table, ids, vocab, top}, n_routes, 0, e_hi, bn, sorted_route, slot_of, expert_offsets, tile_expert,
                      tile_row0, tile_rows, n_tiles, stream);
}

extern "C" int fi_moe_gather(const void* x, const int* sorted_route, const int* expert_offsets, int EL,
                             int n_routes, int K, int H, void* x_sorted, int dtype, void* stream) {
  if (n_routes <= 0) return 0;
  if (H % 8 != 0) return -10;
  if (dtype == 0)
    fi::launch_kernel(moe_gather_kernel<__nv_bfloat16>, dim3(n_routes), dim3(128), 0, FI_STREAM(stream), 0,
                      (const __nv_bfloat16*)x, sorted_route, expert_offsets, EL, K, H, (__nv_bfloat16*)x_sorted);
  else
    fi::launch_kernel(moe_gather_kernel<__half>, dim3(n_routes), dim3(128), 0, FI_STREAM(stream), 0,
                      (const __half*)x, sorted_route, expert_offsets, EL, K, H, (__half*)x_sorted);
  return static_cast<int>(cudaGetLastError());
}

extern "C" int fi_moe_combine(const void* y_sorted, const int* slot_of, const float* topk_w,
                              const void* residual, void* out, int T, int K, int H, int dtype,
                              void* stream) {
  if (T <= 0) return 0;
  if (H % 8 != 0) return -10;
  if (dtype == 0)
    fi::launch_kernel(moe_combine_kernel<__nv_bfloat16>, dim3(T, T < 128 ? (H / 8 + 127) / 128 : 1), dim3(128), 0, FI_STREAM(stream), 0,
                      (const __nv_bfloat16*)y_sorted, slot_of, topk_w, (const __nv_bfloat16*)residual,
                      (__nv_bfloat16*)out, K, H);
  else
    fi::launch_kernel(moe_combine_kernel<__half>, dim3(T, T < 128 ? (H / 8 + 127) / 128 : 1), dim3(128), 0, FI_STREAM(stream), 0,
                      (const __half*)y_sorted, slot_of, topk_w, (const __half*)residual, (__half*)out, K, H);
  return static_cast<int>(cudaGetLastError());
}

// Expert products without tensor cores (dtype 0 bf16, 1 fp16, 2 fp32; any sizes), over the tile table of fi_moe_align
// (built with bn <= 32).  gather != 0: out[row] = silu(Wg x) * (Wu x) (act 1) or, with g = min(Wg x, limit) and
// u = Wu x bounded by limit on both sides, g sigmoid(1.702 g) (u + 1) (act 4), for x = X[sorted_route[row] / top], weights
// [experts, 2 N, K]; gather == 0: out[row] = W X[row], weights [experts, N, K].
extern "C" int fi_moe_expert_rows(const void* x, long ldx, const void* w, void* out, long ldo, const int* sorted_route,
                                  const int* tile_expert, const int* tile_row0, const int* tile_rows, const int* n_tiles,
                                  int max_tiles, int N, int K, int top, int gather, int act, float limit, int dtype,
                                  void* stream) {
  if (max_tiles <= 0) return 0;
  if (gather && act != 1 && act != 4) return -11;
  if (N <= 0 || K <= 0 || top <= 0 || max_tiles > 65535 || (gather && sorted_route == nullptr)) return -10;
  ExpertRows p = {};
  p.x = x; p.w = w; p.out = out; p.ldx = ldx; p.ldo = ldo; p.sorted_route = sorted_route; p.tile_expert = tile_expert;
  p.tile_row0 = tile_row0; p.tile_rows = tile_rows; p.n_tiles = n_tiles; p.N = N; p.K = K; p.top = top; p.gather = gather;
  p.act = act; p.limit = limit;
  const dim3 grid((N + 63) / 64, max_tiles);
  if (dtype == 0) return static_cast<int>(fi::launch_kernel(moe_expert_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, FI_STREAM(stream), 0, p));
  if (dtype == 1) return static_cast<int>(fi::launch_kernel(moe_expert_rows_kernel<__half>, grid, dim3(256), 0, FI_STREAM(stream), 0, p));
  if (dtype == 2) return static_cast<int>(fi::launch_kernel(moe_expert_rows_kernel<float>, grid, dim3(256), 0, FI_STREAM(stream), 0, p));
  return -11;
}
