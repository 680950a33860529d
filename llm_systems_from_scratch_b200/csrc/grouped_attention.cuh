// Sizes and constants shared by the kernels of grouped attention (see grouped_attention.cu).
#pragma once
#include "typed.cuh"

namespace b200 {

// Passed by pointer through the C interface: the field order is part of it.
struct GroupedShape {
  int heads, kv_heads, maps, dim, vdim;
  int qp, kp, vp;               // pitches of a query vector, a cached key, a cached value
  int window;
  float scale, eps, difference, out_scale;
};

inline bool shape_ok(const GroupedShape& s) {
  return s.heads > 0 && s.kv_heads > 0 && s.heads % s.kv_heads == 0 && (s.maps == 1 || s.maps == 2) && s.dim > 0 && s.vdim > 0 &&
         s.qp >= s.kp && s.kp >= s.dim && s.vp >= s.vdim && s.qp % 8 == 0 && s.kp % 8 == 0 && s.vp % 8 == 0 && s.window > 0;
}

}  // namespace b200
