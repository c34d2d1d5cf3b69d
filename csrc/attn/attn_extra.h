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
  // both maps of a head lie in one group of query heads, and the gated form of two maps does not exist
  return p.x.maps == 1 || ((nh / nkv) % 2 == 0 && p.x.gate == nullptr);
}

}  // namespace fi
