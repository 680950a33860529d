// Sizes and constants shared by the kernels of grouped attention (see grouped_attention.cu).
#pragma once
#include "typed.cuh"

namespace b200 {

// Passed by pointer through the C interface: the field order is part of it.
struct GroupedShape {
  int heads, kv_heads, maps, dim, vdim;
  int qp, kp, vp;               // pitches of a query vector, a cached key, a cached value
  int window, keep;             // position i sees j if i - j < window or j < keep; chunked: if i / window == j / window
  float scale, eps, difference, out_scale, softcap;      // softcap 0: none
  const float* sink;            // (heads) or null: exp(sink) joins the denominator (one map)
  const float* slopes;          // (heads) or null: slope * distance comes off the scaled score (one map, no bias table)
  int chunked, head_gate;       // head_gate: the output gate has a column per head, not per element
};

inline bool shape_ok(const GroupedShape& s) {
  return s.heads > 0 && s.kv_heads > 0 && s.heads % s.kv_heads == 0 && (s.maps == 1 || s.maps == 2) && s.dim > 0 && s.vdim > 0 &&
         s.qp >= s.kp && s.kp >= s.dim && s.vp >= s.vdim && s.qp % 8 == 0 && s.kp % 8 == 0 && s.vp % 8 == 0 && s.window > 0 && s.keep >= 0 &&
         s.softcap >= 0.f && (s.sink == nullptr || s.maps == 1) &&
         (s.slopes == nullptr || (s.maps == 1 && s.softcap == 0.f)) && !(s.chunked && s.keep > 0);
}

constexpr float LOG2E = 1.4426950408889634f;

// First position that position pos sees besides the kept ones: that of its window (negative: before the sequence), or of its chunk.
__device__ __forceinline__ int first_seen(const GroupedShape& s, int pos) {
  return s.chunked ? pos - pos % s.window : pos - s.window + 1;
}
// Columns of the output gate in front of head h.
__device__ __forceinline__ int gate_column(const GroupedShape& s, int h) { return s.head_gate ? h : h * s.vdim; }

// cap tanh(x / cap) log2(e) for x = score * scale: tanh(z) = 1 - 2 / (1 + exp(2 z)), whose error is one of rounding in the result's own
// scale.  slope = 2 log2(e) scale / cap, top = cap log2(e).
__device__ __forceinline__ float capped_log2(float score, float slope, float top) {
  return fmaf(-2.f * top, __fdividef(1.f, 1.f + exp2f(score * slope)), top);
}

}  // namespace b200
