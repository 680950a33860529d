// Retention: linear attention with a fixed decay per head.  Per head S_t = decay S_(t-1) + k_t v_t^T and o_t = S_t^T q_t with
// rotated q, k (rotate-half pairs, 32-bit angles) and k scaled by dim^(-1/2); the output of a head is divided by its root
// mean square and multiplied by silu(gate).  The state (heads, dim, vdim) is fp32 and lives in a slot per request.
#include "typed.cuh"

namespace b200 {

struct RetentionParams {
  const void* proj;          // (rows, ld_proj): q | k | v | gate, heads contiguous inside each
  long long ld_proj;
  void* y;                   // (rows, ld_y): gated, normalised heads
  long long ld_y;
  float* state;              // (slots, heads, dim, vdim)
  const int* state_slots;    // per sequence of the launch; negative = padding
  const int* cu;             // optional (seqs + 1): rows of each sequence; null = one row per sequence
  const int* positions;      // per row of the launch
  const float* cos_sin;      // (2, ctx, rot / 2)
  const float* decay;        // (heads)
  int seqs, rows, heads, dim, vdim, rot, ctx, num_slots;
  float eps;
  uint32_t* status;
};

// One block per (sequence, head), tokens in order.  A decode step is the case of one token per sequence: the state is
// read once and written once, with the rotation, the norm and the gate in the same pass.  Longer sequences keep
// the state in global memory (every thread re-reads only what it wrote), so any dim and vdim work.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) retention_recurrent_kernel(const RetentionParams p) {
  pdl_sync();
  extern __shared__ float rsm[];
  __shared__ float red[32];
  const int seq = blockIdx.x, h = blockIdx.y;
  const int D = p.dim, E = p.vdim;
  const int groups = E / VEC;                          // column groups
  const int cgt = groups < 256 ? groups : 256;
  const int rg = 256 / cgt;
  float* qs = rsm;                 // [D]
  float* ks = qs + D;              // [D]
  float* part = ks + D;            // [rg][E]
  const int ty = threadIdx.x / cgt, tx = threadIdx.x - ty * cgt;
  const int row0 = p.cu != nullptr ? p.cu[seq] : seq;
  const int row1 = p.cu != nullptr ? p.cu[seq + 1] : seq + 1;
  const int slot = p.state_slots[seq];
  const T* proj = reinterpret_cast<const T*>(p.proj);
  T* y = reinterpret_cast<T*>(p.y);
  if (slot < 0 || slot >= p.num_slots) {
    if (slot >= p.num_slots && threadIdx.x == 0) report_bad_arg(p.status, 7);
    for (int row = row0; row < row1; ++row)
      for (int c = threadIdx.x; c < E; c += 256) from_f(y[(long long)row * p.ld_y + h * E + c], 0.f);
    return;
  }
  float* S = p.state + ((long long)slot * p.heads + h) * D * E;
  const float decay = p.decay[h];
  const float kscale = rsqrtf((float)D);
  const int half = p.rot / 2;
  for (int row = row0; row < row1; ++row) {
    const T* pr = proj + (long long)row * p.ld_proj;
    const T* qr = pr + h * D;
    const T* kr = pr + p.heads * D + h * D;
    const T* vr = pr + 2 * p.heads * D + h * E;
    const T* gr = pr + 2 * p.heads * D + p.heads * E + h * E;
    int pos = p.positions[row];
    if (pos < 0 || (p.rot > 0 && pos >= p.ctx)) {
      if (threadIdx.x == 0) report_bad_arg(p.status, 8);
      pos = 0;
    }
    for (int d = threadIdx.x; d < D; d += 256) {
      float qv = to_f(qr[d]), kv = to_f(kr[d]);
      if (d < p.rot) {
        const int i = d < half ? d : d - half;
        const float c = p.cos_sin[(long long)pos * half + i], s = p.cos_sin[((long long)p.ctx + pos) * half + i];
        if (d < half) {
          qv = qv * c - to_f(qr[d + half]) * s;
          kv = kv * c - to_f(kr[d + half]) * s;
        } else {
          qv = qv * c + to_f(qr[d - half]) * s;
          kv = kv * c + to_f(kr[d - half]) * s;
        }
      }
      qs[d] = qv;
      ks[d] = kv * kscale;
    }
    __syncthreads();
    const bool fresh = pos == 0;                     // a sequence starts from the zero state, whatever its slot held
    if (ty < rg) {
      for (int g = tx; g < groups; g += cgt) {
        float v[VEC], o[VEC];
        load_vec<VEC>(vr + g * VEC, v);
#pragma unroll
        for (int i = 0; i < VEC; ++i) o[i] = 0.f;
#pragma unroll 8
        for (int d = ty; d < D; d += rg) {
          float s[VEC];
          float* sp = S + (long long)d * E + g * VEC;
          if (fresh) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) s[i] = 0.f;
          } else {
            load_vec<VEC>(sp, s);
          }
          const float kd = ks[d], qd = qs[d];
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            s[i] = fmaf(decay, s[i], kd * v[i]);
            o[i] = fmaf(s[i], qd, o[i]);
          }
          store_vec<VEC>(sp, s);
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) part[ty * E + g * VEC + i] = o[i];
      }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = threadIdx.x; c < E; c += 256) {
      float o = 0.f;
      for (int r = 0; r < rg; ++r) o += part[r * E + c];
      part[c] = o;                                   // row 0 of this column is read by this thread only
      ss += o * o;
    }
    const float inv = rsqrtf(block_total(ss, red) / (float)E + p.eps);
    for (int c = threadIdx.x; c < E; c += 256) {
      const float g = to_f(gr[c]);
      from_f(y[(long long)row * p.ld_y + h * E + c], part[c] * inv * (g / (1.f + expf(-g))));
    }
    __syncthreads();
  }
}

}  // namespace b200

using namespace b200;

// See RetentionParams.  f32 != 0: activations are fp32, else bf16.
extern "C" int b200_retention_recurrent(const void* proj, long long ld_proj, void* y, long long ld_y, float* state,
                                        const int* state_slots, const int* cu, const int* positions, const float* cos_sin,
                                        const float* decay, int seqs, int rows, int heads, int dim, int vdim, int rot,
                                        int ctx, int num_slots, float eps, int f32, uint32_t* status, cudaStream_t st) {
  if (seqs <= 0 || rows <= 0) return 0;
  if (heads <= 0 || dim <= 0 || vdim <= 0 || rot < 0 || rot > dim || (rot & 1) || (rot > 0 && cos_sin == nullptr) ||
      heads > 65535)
    return -10;
  RetentionParams p;
  p.proj = proj; p.ld_proj = ld_proj; p.y = y; p.ld_y = ld_y; p.state = state; p.state_slots = state_slots; p.cu = cu;
  p.positions = positions; p.cos_sin = cos_sin; p.decay = decay; p.seqs = seqs; p.rows = rows; p.heads = heads;
  p.dim = dim; p.vdim = vdim; p.rot = rot; p.ctx = ctx; p.num_slots = num_slots; p.eps = eps; p.status = status;
  const bool vec = vdim % 4 == 0 && ld_proj % 4 == 0 && (2 * heads * dim) % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(proj) & 15) == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
  const int groups = vec ? vdim / 4 : vdim;
  const int rg = groups < 256 ? 256 / groups : 1;
  const size_t smem = (2ull * dim + (size_t)rg * vdim) * sizeof(float);
  if (smem > 48 * 1024) return -12;
  const dim3 grid(seqs, heads);
  if (f32) {
    if (vec) launch_dep(retention_recurrent_kernel<float, 4>, grid, 256, smem, st, p);
    else launch_dep(retention_recurrent_kernel<float, 1>, grid, 256, smem, st, p);
  } else {
    if (vec) launch_dep(retention_recurrent_kernel<__nv_bfloat16, 4>, grid, 256, smem, st, p);
    else launch_dep(retention_recurrent_kernel<__nv_bfloat16, 1>, grid, 256, smem, st, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
