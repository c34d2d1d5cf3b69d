// Optional parts of an attention layer that the paged kernels apply themselves (a null pointer: none of them).
#pragma once

extern "C" struct FiAttnExtra {
  const float* sinks;     // fp32 [nh] or null: one extra exp(sink) per head in the softmax denominator
  const void* gate;       // output gate in the type of the output or null: out is multiplied by sigmoid(gate)
  long gate_stride;       // row pitch of gate
  int out_dim;            // channels of a head that are stored (0 = head size)
  int gate_per_head;      // 0: gate has the channels of the output, 1: one number per head
  int maps;               // 1, or 2: query heads 2 j and 2 j + 1 are the two maps of output head j (see below)
  float lambda;           // maps == 2:  o = a1 - lambda a2,  out_j = o / sqrt(mean(o^2) + eps) * out_scale
  float out_scale;        //             (the mean runs over the out_dim channels; out has nh / 2 heads)
  float eps;
  // Weights without a softmax: a key's weight is sigmoid(score + bias[head]), not divided by anything.
  const float* bias;      // fp32 [nh] or null (softmax); no sinks, gates or two maps beside it
  const float* turn;      // fp32 [turn_rows, out_dim] or null: rows [cos | sin] per position; channels 2 i and 2 i + 1 of the
                          // output turn back by angle i of the query's position before they are stored
  int turn_rows;
  int chunk;              // > 0 (with bias): position i sees keys from floor(i / chunk) * chunk on
};

namespace fi {

// Copies the extras into a kernel's parameters; false when they do not fit nh query heads on nkv key / value heads.
template <typename P>
inline bool take_extra(P& p, const FiAttnExtra* e, int hd, int nh, int nkv) {
  FiAttnExtra none = {};
  none.maps = 1;
  p.x = e != nullptr ? *e : none;
  if (p.x.out_dim == 0) p.x.out_dim = hd;
  if (p.x.out_dim < 0 || p.x.out_dim > hd || p.x.maps < 1 || p.x.maps > 2) return false;
  if (p.x.bias == nullptr && (p.x.turn != nullptr || p.x.chunk != 0)) return false;
  if (p.x.bias != nullptr && (p.x.maps != 1 || p.x.sinks != nullptr || p.x.gate != nullptr || p.x.chunk < 0 || (p.x.out_dim & 1) != 0 ||
                              (p.x.turn != nullptr && p.x.turn_rows <= 0)))
    return false;
  // both maps of a head lie in one group of query heads, and the gated form of two maps does not exist
  return p.x.maps == 1 || ((nh / nkv) % 2 == 0 && p.x.gate == nullptr);
}

#ifdef __CUDACC__
// First key that position pos sees (weights without a softmax: chunks, or the window).
template <typename P>
__device__ __forceinline__ int first_key(const P& p, int pos) {
  if (p.x.chunk > 0) return pos / p.x.chunk * p.x.chunk;
  return p.window > 0 && pos >= p.window ? pos - p.window + 1 : 0;
}
__device__ __forceinline__ float sigmoid_weight(float score) { return __fdividef(1.f, 1.f + __expf(-score)); }
// Channels (u, v) = (2 i, 2 i + 1) of an output turned back by position pos.
template <typename P>
__device__ __forceinline__ void turn_back(const P& p, int pos, int i, float& u, float& v) {
  const float* row = p.x.turn + static_cast<long>(pos < 0 ? 0 : pos >= p.x.turn_rows ? p.x.turn_rows - 1 : pos) * p.x.out_dim;
  const float c = row[i], s = row[p.x.out_dim / 2 + i], a = u;
  u = a * c + v * s;
  v = v * c - a * s;
}
// The same for pairs i .. i + 3 (channels y[0] .. y[7]); i is a multiple of four, and so is out_dim / 2.
template <typename P>
__device__ __forceinline__ void turn_back4(const P& p, int pos, int i, float* y) {
  const float* row = p.x.turn + static_cast<long>(pos < 0 ? 0 : pos >= p.x.turn_rows ? p.x.turn_rows - 1 : pos) * p.x.out_dim + i;
  const float4 c4 = *reinterpret_cast<const float4*>(row), s4 = *reinterpret_cast<const float4*>(row + p.x.out_dim / 2);
  const float c[4] = {c4.x, c4.y, c4.z, c4.w}, s[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float u = y[2 * e], v = y[2 * e + 1];
    y[2 * e] = u * c[e] + v * s[e];
    y[2 * e + 1] = v * c[e] - u * s[e];
  }
}
#endif

}  // namespace fi
