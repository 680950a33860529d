// Kernels around the mixers of a layered decoder with a 32-bit residual stream: embedding / residual update / RMS norm /
// expert scatter in one pass over a row, the plan of a token-table mixture of experts, and small element-wise steps.
// T is the activation type: bf16 when serving, fp32 when a model runs in 32-bit.
#include "typed.cuh"

namespace b200 {

struct ResidualNormParams {
  // source of the row: the embedding table times embed_scale (tokens != null, written to x) or x itself
  const long long* tokens;
  const void* embed;
  int vocab;
  float embed_scale;
  float* x;                  // (rows, d) fp32 residual stream
  const long long* row_index;  // optional: output row i reads residual row row_index[i] and x is not written
  // optional expert outputs that belong to the row: x += yscale * sum_k yweight[row, k] * y[ypos[row, k]] (yweight null: ones).
  // A choice with ypos = -2 stands for the experts' input z[row] itself; s[row], times sigmoid(sgate[row]), is an expert's output
  // that every row receives.
  const void* y;
  const int* ypos;
  const float* yweight;
  int ytop, y_rows;
  float yscale;
  long long ld_y;
  const void *z, *s;
  const float* sgate;
  long long ld_z, ld_s, ld_sgate;
  // norm: h = x / rms(x) * (w + w_offset) (h == null: only the residual is updated)
  const void* w;
  float w_offset;
  void* h;
  long long ld_h;
  float eps;
  // optional copies of the normed row at the places its experts read: xg[gpos[row, k]] = h
  void* xg;
  const int* gpos;
  int gtop, xg_rows;
  long long ld_xg;
  int rows, x_rows, d;
  uint32_t* status;
};

// One block per row.  A thread keeps KEEP groups of its columns in registers between the passes, and requests all of them before it
// works on the first; columns of wider rows are read (and, where experts add to a row that is not stored, added up) again.
template <typename T, int VEC>
__global__ void __launch_bounds__(256, 3) residual_norm_kernel(const ResidualNormParams p) {
  pdl_sync();
  __shared__ float red[32];
  const int row = blockIdx.x;
  long long src = row;
  if (p.row_index != nullptr) {
    src = p.row_index[row];
    if (src < 0 || src >= p.x_rows) {
      if (threadIdx.x == 0) report_bad_arg(p.status, 1);
      src = 0;
    }
  }
  float* xr = p.x + src * p.d;
  const T* er = nullptr;
  if (p.tokens != nullptr) {
    long long tok = p.tokens[row];
    if (tok < 0 || tok >= p.vocab) {
      if (threadIdx.x == 0) report_bad_arg(p.status, 2);
      tok = 0;
    }
    er = reinterpret_cast<const T*>(p.embed) + tok * p.d;
  }
  const bool changed = (er != nullptr || p.y != nullptr) && p.row_index == nullptr;
  const float share = p.s != nullptr ? (p.sgate != nullptr ? 1.f / (1.f + expf(-p.sgate[src * p.ld_sgate])) : 1.f) : 0.f;
  constexpr int KEEP = 4;
  const int step = blockDim.x * VEC, c0 = threadIdx.x * VEC;
  // columns of the first GROUPS groups, from c on, as the sublayers have left them
  auto gather = [&](int c, auto& f) __attribute__((always_inline)) {
    constexpr int GROUPS = sizeof(f) / sizeof(f[0]);
#pragma unroll
    for (int j = 0; j < GROUPS; ++j) {
      if (c + j * step >= p.d) break;
      if (er != nullptr) {
        load_vec<VEC>(er + c + j * step, f[j]);
#pragma unroll
        for (int i = 0; i < VEC; ++i) f[j][i] *= p.embed_scale;
      } else {
        load_vec<VEC>(xr + c + j * step, f[j]);
      }
    }
    if (p.y == nullptr) return;
    auto add = [&](const T* from, float a) __attribute__((always_inline)) {
      float g[GROUPS][VEC];
#pragma unroll
      for (int j = 0; j < GROUPS; ++j)
        if (c + j * step < p.d) load_vec<VEC>(from + c + j * step, g[j]);
#pragma unroll
      for (int j = 0; j < GROUPS; ++j)
#pragma unroll
        for (int i = 0; i < VEC; ++i) f[j][i] = fmaf(a, g[j][i], f[j][i]);
    };
    if (p.s != nullptr) add(reinterpret_cast<const T*>(p.s) + src * p.ld_s, p.yscale * share);
#pragma unroll 1
    for (int k = 0; k < p.ytop; ++k) {
      const int pos = p.ypos[src * p.ytop + k];
      const float a = p.yscale * (p.yweight != nullptr ? p.yweight[src * p.ytop + k] : 1.f);
      if (pos >= 0 && pos < p.y_rows) add(reinterpret_cast<const T*>(p.y) + (long long)pos * p.ld_y, a);
      else if (pos == -2 && p.z != nullptr) add(reinterpret_cast<const T*>(p.z) + src * p.ld_z, a);
      // else: a padding row of the batch
    }
  };
  float keep[KEEP][VEC], ss = 0.f;
  gather(c0, keep);
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    if (c0 + j * step >= p.d) break;
    if (changed) store_vec<VEC>(xr + c0 + j * step, keep[j]);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(keep[j][i], keep[j][i], ss);
  }
  for (int c = c0 + KEEP * step; c < p.d; c += step) {
    float f[1][VEC];
    gather(c, f);
    if (changed) store_vec<VEC>(xr + c, f[0]);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(f[0][i], f[0][i], ss);
  }
  if (p.h == nullptr) return;
  const T* w = reinterpret_cast<const T*>(p.w);
  Raw<T, VEC> wk[KEEP];                      // requested before the block waits for its sum
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if (c0 + j * step < p.d) wk[j] = *reinterpret_cast<const Raw<T, VEC>*>(w + c0 + j * step);
  const float r = rsqrtf(block_total(ss, red) / (float)p.d + p.eps);
  T* hr = reinterpret_cast<T*>(p.h) + (long long)row * p.ld_h;
  auto finish = [&](int c, const Raw<T, VEC>& wr, float (&f)[VEC]) __attribute__((always_inline)) {
    float g[VEC];
    load_vec<VEC>(wr.v, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) f[i] = f[i] * r * (g[i] + p.w_offset);
    store_vec<VEC>(hr + c, f);
    if (p.xg != nullptr) {
      for (int k = 0; k < p.gtop; ++k) {
        const int pos = p.gpos[(long long)row * p.gtop + k];
        if (pos >= 0 && pos < p.xg_rows) store_vec<VEC>(reinterpret_cast<T*>(p.xg) + (long long)pos * p.ld_xg + c, f);
      }
    }
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if (c0 + j * step < p.d) finish(c0 + j * step, wk[j], keep[j]);
  for (int c = c0 + KEEP * step; c < p.d; c += step) {
    float f[1][VEC];
    if (changed) load_vec<VEC>(xr + c, f[0]);
    else gather(c, f);
    finish(c, *reinterpret_cast<const Raw<T, VEC>*>(w + c), f[0]);
  }
}

// Norms behind the sublayers: x += y / rms(y) * w for a sublayer's output y, and h = x in the activation type, which the next
// sublayer reads.  With `tokens` the row starts: x = embed[token].  One block per row; a thread keeps its columns of y and x in
// registers between the passes (KEEP groups; wider rows are read again).
struct AddNormedParams {
  const long long* tokens;
  const void *embed, *y, *w;
  float* x;
  void* h;
  int vocab, d;
  long long ld_y, ld_h;
  float eps;
  uint32_t* status;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(256) add_normed_kernel(const AddNormedParams p) {
  pdl_sync();
  __shared__ float red[32];
  const long long row = blockIdx.x;
  float* xr = p.x + row * p.d;
  T* hr = reinterpret_cast<T*>(p.h) + row * p.ld_h;
  if (p.tokens != nullptr) {
    long long tok = p.tokens[row];
    if (tok < 0 || tok >= p.vocab) {
      if (threadIdx.x == 0) report_bad_arg(p.status, 20);
      tok = 0;
    }
    const T* er = reinterpret_cast<const T*>(p.embed) + tok * p.d;
    for (int c = threadIdx.x * VEC; c < p.d; c += blockDim.x * VEC) {
      float f[VEC];
      load_vec<VEC>(er + c, f);
      store_vec<VEC>(xr + c, f);
      store_vec<VEC>(hr + c, f);
    }
    return;
  }
  const T* yr = reinterpret_cast<const T*>(p.y) + row * p.ld_y;
  const T* w = reinterpret_cast<const T*>(p.w);
  constexpr int KEEP = 4;
  float y[KEEP][VEC], x[KEEP][VEC];
  const int step = blockDim.x * VEC;
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x * VEC + j * step;
    if (c < p.d) {
      load_vec<VEC>(yr + c, y[j]);
      load_vec<VEC>(xr + c, x[j]);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss += y[j][i] * y[j][i];
    }
  }
  for (int c = threadIdx.x * VEC + KEEP * step; c < p.d; c += step) {
    float f[VEC];
    load_vec<VEC>(yr + c, f);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += f[i] * f[i];
  }
  const float r = rsqrtf(block_total(ss, red) / (float)p.d + p.eps);
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x * VEC + j * step;
    if (c < p.d) {
      float g[VEC];
      load_vec<VEC>(w + c, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[j][i] += y[j][i] * r * g[i];
      store_vec<VEC>(xr + c, x[j]);
      store_vec<VEC>(hr + c, x[j]);
    }
  }
  for (int c = threadIdx.x * VEC + KEEP * step; c < p.d; c += step) {
    float f[VEC], g[VEC], v[VEC];
    load_vec<VEC>(yr + c, f);
    load_vec<VEC>(xr + c, v);
    load_vec<VEC>(w + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] += f[i] * r * g[i];
    store_vec<VEC>(xr + c, v);
    store_vec<VEC>(hr + c, v);
  }
}

// -------------------------------------------------------------------------------------------------- mixture of experts
// Plan of a mixture of experts whose experts are looked up by token id: sort the (row, choice) pairs by expert into
// 128-row tiles that each belong to one expert.  One block per layer (every layer has its own table).
//   pos[row, k]       row of the expert-sorted buffers that choice k of `row` uses (-1: a padding row of the batch)
//   tile_group[t]     expert of row tile t, -1 = tile not used
constexpr int PLAN_LAYERS = 48;
constexpr int PLAN_TILE = 128;
struct MoePlanParams {
  const long long* tokens;
  const long long* slots;      // negative = padding row
  int rows, vocab;
  const int* table[PLAN_LAYERS];
  int experts[PLAN_LAYERS], top[PLAN_LAYERS];
  int* pos;
  long long pos_stride;        // ints between layers
  int* tile_group;
  int tile_stride;             // tiles per layer
  uint32_t* status;
};

// Adds 1 to counter[e] for every lane with e >= 0 and returns the lane's ticket; one atomic per distinct e and warp.
__device__ __forceinline__ int warp_ticket(int* counter, int e) {
  const uint32_t peers = __match_any_sync(0xffffffffu, e);
  const int lane = threadIdx.x & 31, leader = __ffs(peers) - 1;
  int base = 0;
  if (lane == leader && e >= 0) base = atomicAdd(&counter[e], __popc(peers));
  base = __shfl_sync(0xffffffffu, base, leader);
  return base + __popc(peers & ((1u << lane) - 1u));
}

__global__ void __launch_bounds__(1024) moe_plan_kernel(const MoePlanParams p) {
  pdl_sync();
  extern __shared__ int plan_smem[];
  const int layer = blockIdx.x;
  const int E = p.experts[layer], top = p.top[layer];
  int* count = plan_smem;          // [E]
  int* next = plan_smem + E;       // [E] first free row of the expert's tiles
  int* used = plan_smem + 2 * E;   // [1] tiles in use
  const int* table = p.table[layer];
  int* pos = p.pos + layer * p.pos_stride;
  int* groups = p.tile_group + (long long)layer * p.tile_stride;
  for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = 0;
  __syncthreads();
  const int items = p.rows * top;
  const int items_up = (items + (int)blockDim.x - 1) / (int)blockDim.x * (int)blockDim.x;
  auto expert_of = [&](int i) -> int {
    if (i >= items) return -1;
    const int row = i / top;
    if (p.slots[row] < 0) return -1;
    const long long tok = p.tokens[row];
    if (tok < 0 || tok >= p.vocab) return -1;
    const int e = table[tok * top + (i - row * top)];
    if (e < 0 || e >= E) {
      report_bad_arg(p.status, 3);
      return -1;
    }
    return e;
  };
  for (int i = threadIdx.x; i < items_up; i += blockDim.x) warp_ticket(count, expert_of(i));
  __syncthreads();
  if (threadIdx.x == 0) {
    int tile = 0;
    for (int e = 0; e < E; ++e) {
      next[e] = tile * PLAN_TILE;
      tile += (count[e] + PLAN_TILE - 1) / PLAN_TILE;
    }
    *used = tile;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    const int t0 = next[e] / PLAN_TILE, nt = (count[e] + PLAN_TILE - 1) / PLAN_TILE;
    for (int t = t0; t < t0 + nt && t < p.tile_stride; ++t) groups[t] = e;
  }
  for (int t = *used + threadIdx.x; t < p.tile_stride; t += blockDim.x) groups[t] = -1;
  __syncthreads();
  for (int i = threadIdx.x; i < items_up; i += blockDim.x) {
    const int e = expert_of(i);
    const int at = warp_ticket(next, e);
    if (i < items) pos[i] = e >= 0 && at < p.tile_stride * PLAN_TILE ? at : -1;
  }
}

// h = act(gate) * up for gu (rows, 2F), gate columns first; any F, any row pitch.  act: silu, or relu.
template <typename T>
__global__ void glu_any_kernel(const T* __restrict__ gu, T* __restrict__ h, long long rows, int F, long long ld_gu,
                               long long ld_h, int relu) {
  pdl_sync();
  const long long n = rows * F;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / F;
    const int c = (int)(i - r * F);
    const float g = to_f(gu[r * ld_gu + c]), u = to_f(gu[r * ld_gu + F + c]);
    from_f(h[r * ld_h + c], (relu ? fmaxf(g, 0.f) : g / (1.f + expf(-g))) * u);
  }
}

// o *= sigmoid(g), a gate for every `per` columns.
template <typename T>
__global__ void gate_sigmoid_kernel(T* __restrict__ o, const T* __restrict__ g, long long rows, int n, int per, long long ld_o,
                                    long long ld_g) {
  pdl_sync();
  const long long total = rows * n;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / n;
    const int c = (int)(i - r * n);
    const float s = 1.f / (1.f + expf(-to_f(g[r * ld_g + c / per])));
    from_f(o[r * ld_o + c], to_f(o[r * ld_o + c]) * s);
  }
}

static int blocks_for(long long work, int threads) {
  long long b = (work + threads - 1) / threads;
  if (b < 1) b = 1;
  return (int)(b > 148 * 16 ? 148 * 16 : b);
}

}  // namespace b200

using namespace b200;

// What the experts add, passed by pointer through the C interface: the field order is part of it.
struct ExpertOutputs {
  const void* y;
  const int* ypos;
  const float* yweight;
  const void *z, *s;
  const float* sgate;
  long long ld_y, ld_z, ld_s, ld_sgate;
  int ytop, y_rows;
  float yscale;
};

// See ResidualNormParams.  f32 != 0: T = float, else bf16.
extern "C" int b200_residual_norm(const long long* tokens, const void* embed, int vocab, float embed_scale, float* x,
                                  const long long* row_index, const ExpertOutputs* ex, const void* w, float w_offset, void* h,
                                  long long ld_h, float eps, void* xg, const int* gpos, int gtop, int xg_rows, long long ld_xg,
                                  int rows, int x_rows, int d, int f32, uint32_t* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (d <= 0 || x == nullptr || (h != nullptr && w == nullptr) || (tokens != nullptr && embed == nullptr) ||
      (ex != nullptr && (ex->y == nullptr || ex->ypos == nullptr)) || (xg != nullptr && (gpos == nullptr || h == nullptr)) ||
      (tokens != nullptr && row_index != nullptr))
    return -10;
  ResidualNormParams p = {};
  p.tokens = tokens; p.embed = embed; p.vocab = vocab; p.embed_scale = embed_scale; p.x = x; p.row_index = row_index;
  if (ex != nullptr) {
    p.y = ex->y; p.ypos = ex->ypos; p.yweight = ex->yweight; p.ytop = ex->ytop; p.y_rows = ex->y_rows; p.yscale = ex->yscale;
    p.ld_y = ex->ld_y; p.z = ex->z; p.ld_z = ex->ld_z; p.s = ex->s; p.ld_s = ex->ld_s; p.sgate = ex->sgate; p.ld_sgate = ex->ld_sgate;
  }
  p.w = w; p.w_offset = w_offset; p.h = h; p.ld_h = ld_h; p.eps = eps;
  p.xg = xg; p.gpos = gpos; p.gtop = gtop; p.xg_rows = xg_rows; p.ld_xg = ld_xg;
  p.rows = rows; p.x_rows = x_rows; p.d = d; p.status = status;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(embed) | reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(p.y) |
                         reinterpret_cast<uintptr_t>(p.z) | reinterpret_cast<uintptr_t>(p.s) | reinterpret_cast<uintptr_t>(w) |
                         reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(xg);
  const bool vec = d % 4 == 0 && (p.ld_y | p.ld_z | p.ld_s | ld_h | ld_xg) % 4 == 0 && (ptrs & 15) == 0;
  const int groups = rows >= 148 * 8 ? 4 : 1;        // of a thread: many rows share an SM, few have all of its threads
  const int per = (vec ? 4 : 1) * groups;
  int threads = ((d + per - 1) / per + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  if (f32) {
    if (vec) launch_dep(residual_norm_kernel<float, 4>, rows, threads, 0, st, p);
    else launch_dep(residual_norm_kernel<float, 1>, rows, threads, 0, st, p);
  } else {
    if (vec) launch_dep(residual_norm_kernel<__nv_bfloat16, 4>, rows, threads, 0, st, p);
    else launch_dep(residual_norm_kernel<__nv_bfloat16, 1>, rows, threads, 0, st, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

extern "C" int b200_moe_plan_layers(void) { return PLAN_LAYERS; }

// tables / experts / top: host arrays of `layers` entries (at most b200_moe_plan_layers()).
extern "C" int b200_moe_plan(const long long* tokens, const long long* slots, int rows, int vocab, int layers,
                             const int* const* tables, const int* experts, const int* top, int* pos, long long pos_stride,
                             int* tile_group, int tile_stride, uint32_t* status, cudaStream_t st) {
  if (rows <= 0 || layers <= 0) return 0;
  if (layers > PLAN_LAYERS || tile_stride <= 0) return -10;
  MoePlanParams p;
  p.tokens = tokens; p.slots = slots; p.rows = rows; p.vocab = vocab;
  p.pos = pos; p.pos_stride = pos_stride; p.tile_group = tile_group; p.tile_stride = tile_stride; p.status = status;
  int emax = 0, tmax = 0;
  for (int i = 0; i < layers; ++i) {
    if (experts[i] <= 0 || top[i] <= 0 || tables[i] == nullptr || (long long)rows * top[i] > pos_stride) return -11;
    p.table[i] = tables[i]; p.experts[i] = experts[i]; p.top[i] = top[i];
    emax = experts[i] > emax ? experts[i] : emax;
    tmax = top[i] > tmax ? top[i] : tmax;
  }
  if (emax > 4096) return -12;
  int threads = (rows * tmax + 31) / 32 * 32;
  if (threads > 1024) threads = 1024;
  launch_dep(moe_plan_kernel, layers, threads, (2 * emax + 1) * sizeof(int), st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// y: (rows, ld_y) sublayer output to norm and add, or tokens / embed to start the rows.  See AddNormedParams.
extern "C" int b200_add_normed(const long long* tokens, const void* embed, int vocab, float* x, const void* y, long long ld_y,
                               const void* w, void* h, long long ld_h, float eps, int rows, int d, int f32, uint32_t* status,
                               cudaStream_t st) {
  if (rows <= 0) return 0;
  if (d <= 0 || x == nullptr || h == nullptr || (tokens != nullptr ? embed == nullptr : (y == nullptr || w == nullptr))) return -10;
  AddNormedParams p;
  p.tokens = tokens; p.embed = embed; p.vocab = vocab; p.x = x; p.y = y; p.ld_y = ld_y; p.w = w; p.h = h; p.ld_h = ld_h;
  p.eps = eps; p.d = d; p.status = status;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(embed) | reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(y) |
                         reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(h);
  const bool vec = d % 4 == 0 && ld_y % 4 == 0 && ld_h % 4 == 0 && (ptrs & 15) == 0;
  const int per = vec ? 8 : 2;                       // two groups per thread
  int threads = ((d + per - 1) / per + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  if (f32) {
    if (vec) launch_dep(add_normed_kernel<float, 4>, rows, threads, 0, st, p);
    else launch_dep(add_normed_kernel<float, 1>, rows, threads, 0, st, p);
  } else {
    if (vec) launch_dep(add_normed_kernel<__nv_bfloat16, 4>, rows, threads, 0, st, p);
    else launch_dep(add_normed_kernel<__nv_bfloat16, 1>, rows, threads, 0, st, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

extern "C" int b200_glu_any(const void* gu, void* h, long long rows, int F, long long ld_gu, long long ld_h, int relu, int f32,
                            cudaStream_t st) {
  if (rows <= 0) return 0;
  const int g = blocks_for(rows * F, 256);
  if (f32) launch_dep(glu_any_kernel<float>, g, 256, 0, st, (const float*)gu, (float*)h, rows, F, ld_gu, ld_h, relu);
  else
    launch_dep(glu_any_kernel<__nv_bfloat16>, g, 256, 0, st, (const __nv_bfloat16*)gu, (__nv_bfloat16*)h, rows, F, ld_gu, ld_h,
               relu);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

extern "C" int b200_gate_sigmoid(void* o, const void* g, long long rows, int n, int per, long long ld_o, long long ld_g, int f32,
                                 cudaStream_t st) {
  if (rows <= 0) return 0;
  if (per <= 0) return -10;
  const int b = blocks_for(rows * n, 256);
  if (f32) launch_dep(gate_sigmoid_kernel<float>, b, 256, 0, st, (float*)o, (const float*)g, rows, n, per, ld_o, ld_g);
  else
    launch_dep(gate_sigmoid_kernel<__nv_bfloat16>, b, 256, 0, st, (__nv_bfloat16*)o, (const __nv_bfloat16*)g, rows, n,
               per, ld_o, ld_g);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
