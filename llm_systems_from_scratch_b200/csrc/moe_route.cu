// Mixture of experts with a learned router: choice of experts per row, then the rows sorted by expert into 128-row tiles.
//
// The router's logits come out of a GEMM in fp32, or, for the few rows of a decode step, out of moe_route_rows itself (one block per row).
// moe_route takes the softmax over all outputs of a row, chooses the `top` outputs
// with the largest score + correction (without a correction: the largest logits) and weighs them with their share of the scores, which is the
// softmax over the chosen logits; a bias may be added to the logits first; outputs from `experts` on are identities (the
// experts' input itself) and need no expert row.  A chosen expert's place among the rows that chose it comes from a counter per
// expert (counted per block in shared memory first).  moe_dispatch turns the counters into tiles (every block does the short prefix
// sum itself), writes where each choice's row went and copies the rows there.  `always` further experts behind the others receive every
// row (a shared expert in pieces of the experts' size), weighted by the sigmoid of one more logit.  Which row of a tile a token gets depends on the
// order of the atomics; what is computed for it does not.
#include "typed.cuh"

namespace b200 {

constexpr int ROUTE_TILE = 128;            // rows of an expert tile (mixer_elementwise.cu: PLAN_TILE)
constexpr int ROUTE_WARPS = 8;
constexpr int ROUTE_ROWS = 4;              // rows of a warp

struct RouteParams {
  const float* z;              // (rows, ld_z): logits of experts + identities
  long long ld_z;
  const float* bias;           // (outputs) added to the logits, or null
  const float* correction;     // (outputs), or null: the choice is by logit
  const long long* slots;      // negative = padding row
  int* choice;                 // (rows, top): chosen output, -1 for a padding row
  int* rank;                   // (rows, top): place among the rows of the chosen expert
  float* weight;               // (rows, top + always)
  int* count;                  // (experts), zero before the launch
  int rows, experts, outputs, top, always;       // always > 0: z has one more column
};

// Choice of one row by one warp: the softmax of s[0 .. outputs) (plus bias) in place, then outputs with the largest score + correction, which go to
// picked[0], picked[stride], ...  Returns the sum of the chosen scores.  key: scratch.  Ties go to the lower index.
__device__ __forceinline__ float route_choose(float* s, float* key, const float* __restrict__ bias, const float* __restrict__ correction, int outputs,
                                              int top, int* picked, int stride) {
  const int lane = threadIdx.x & 31;
  float mx = -INFINITY;
  for (int e = lane; e < outputs; e += 32) {
    if (bias != nullptr) s[e] += bias[e];
    mx = fmaxf(mx, s[e]);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
  float sum = 0.f;
  for (int e = lane; e < outputs; e += 32) {
    key[e] = s[e];
    sum += s[e] = expf(s[e] - mx);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  for (int e = lane; e < outputs; e += 32) {
    s[e] /= sum;
    if (correction != nullptr) key[e] = s[e] + correction[e];
  }
  __syncwarp();
  float total = 0.f;
  for (int k = 0; k < top; ++k) {            // a lane looks after outputs lane, lane + 32, ...
    float best = -INFINITY;
    int at = outputs;
    for (int e = lane; e < outputs; e += 32)
      if (key[e] > best) {
        best = key[e];
        at = e;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (ob > best || (ob == best && oa < at)) {
        best = ob;
        at = oa;
      }
    }
    if (at >= outputs) at = 0;               // not a number anywhere: something valid
    total += s[at];
    if (lane == (at & 31)) key[at] = -INFINITY;
    if (lane == 0) picked[k * stride] = at;
  }
  __syncwarp();
  return total;
}

// One warp per row at a time; shared memory: per warp the scores and the choice scores, per block a counter and a base per expert.
__global__ void __launch_bounds__(ROUTE_WARPS * 32) moe_route_kernel(const RouteParams p) {
  pdl_sync();
  extern __shared__ float rsm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* s = rsm + warp * 2 * p.outputs;
  float* key = s + p.outputs;
  int* local = reinterpret_cast<int*>(rsm + ROUTE_WARPS * 2 * p.outputs);
  int* base = local + p.experts;
  int* picked = base + p.experts;            // [ROUTE_WARPS * ROUTE_ROWS][top][2]: expert, place within the block
  for (int e = threadIdx.x; e < p.experts; e += blockDim.x) local[e] = 0;
  __syncthreads();
  const int row0 = (blockIdx.x * ROUTE_WARPS + warp) * ROUTE_ROWS;
  for (int r = 0; r < ROUTE_ROWS && row0 + r < p.rows; ++r) {
    const int row = row0 + r;
    int* mine = picked + (warp * ROUTE_ROWS + r) * p.top * 2;
    if (p.slots[row] < 0) {
      for (int k = lane; k < p.top; k += 32) {
        mine[2 * k] = -1;
        p.choice[(long long)row * p.top + k] = -1;
        p.weight[(long long)row * (p.top + p.always) + k] = 0.f;
      }
      for (int k = lane; k < p.always; k += 32) p.weight[(long long)row * (p.top + p.always) + p.top + k] = 0.f;
      continue;
    }
    const float* z = p.z + (long long)row * p.ld_z;
    for (int e = lane; e < p.outputs; e += 32) s[e] = z[e];
    const float total = route_choose(s, key, p.bias, p.correction, p.outputs, p.top, mine, 2);
    for (int k = lane; k < p.top; k += 32)
      if (mine[2 * k] < p.experts) mine[2 * k + 1] = atomicAdd(&local[mine[2 * k]], 1);
    for (int k = lane; k < p.top; k += 32) {
      p.choice[(long long)row * p.top + k] = mine[2 * k];
      p.weight[(long long)row * (p.top + p.always) + k] = s[mine[2 * k]] / (total + 1e-20f);
    }
    for (int k = lane; k < p.always; k += 32) p.weight[(long long)row * (p.top + p.always) + p.top + k] = 1.f / (1.f + expf(-z[p.outputs]));
    __syncwarp();
  }
  __syncthreads();
  for (int e = threadIdx.x; e < p.experts; e += blockDim.x) base[e] = local[e] > 0 ? atomicAdd(&p.count[e], local[e]) : 0;
  __syncthreads();
  const int first = blockIdx.x * ROUTE_WARPS * ROUTE_ROWS;
  const int n = min(ROUTE_WARPS * ROUTE_ROWS, p.rows - first) * p.top;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int e = picked[2 * i];
    p.rank[(long long)first * p.top + i] = e >= 0 && e < p.experts ? base[e] + picked[2 * i + 1] : -1;
  }
}

// The same with the logits: z[row] = w h[row] for `columns` rows of w, one block per row.
struct RouteRowsParams {
  RouteParams r;               // z is written here
  float* z;
  const void *h, *w;           // (rows, ld_h), (columns, ld_w)
  long long ld_h, ld_w;
  int d, columns;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(512) moe_route_rows_kernel(const RouteRowsParams p) {
  pdl_sync();
  extern __shared__ float rsm[];
  const RouteParams& r = p.r;
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* s = rsm;                            // [columns] logits
  float* key = s + p.columns;                // [outputs]
  int* picked = reinterpret_cast<int*>(key + r.outputs);       // [top]
  float* hs = rsm + (p.columns + r.outputs + r.top + 3) / 4 * 4;                 // [d] the row
  const T* h = reinterpret_cast<const T*>(p.h) + (long long)row * p.ld_h;
  constexpr int AHEAD = 16;                  // pieces of a router row that a lane requests at a time
  Raw<T, VEC> u[AHEAD];
  auto request = [&](int e, int c0) __attribute__((always_inline)) {
    const T* w = reinterpret_cast<const T*>(p.w) + (long long)e * p.ld_w;
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      const int c = c0 + (j * 32 + lane) * VEC;
      if (c < p.d) u[j] = *reinterpret_cast<const Raw<T, VEC>*>(w + c);
    }
  };
  if (warp < p.columns) request(warp, 0);
  for (int c = threadIdx.x * VEC; c < p.d; c += blockDim.x * VEC) {
    float x[VEC];
    load_vec<VEC>(h + c, x);
    store_vec<VEC>(hs + c, x);
  }
  __syncthreads();
  for (int e = warp; e < p.columns; e += 16) {
    float a = 0.f;
    for (int c0 = 0; c0 < p.d; c0 += 32 * VEC * AHEAD) {
      if (e != warp || c0 > 0) request(e, c0);
#pragma unroll
      for (int j = 0; j < AHEAD; ++j) {
        const int c = c0 + (j * 32 + lane) * VEC;
        if (c < p.d) {
          float x[VEC], y[VEC];
          load_vec<VEC>(hs + c, x);
          load_vec<VEC>(u[j].v, y);
#pragma unroll
          for (int i = 0; i < VEC; ++i) a = fmaf(x[i], y[i], a);
        }
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
    if (lane == 0) s[e] = a;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < p.columns; e += blockDim.x) p.z[(long long)row * r.ld_z + e] = s[e];
  __syncthreads();                           // route_choose overwrites the logits
  if (warp > 0) return;
  const bool live = r.slots[row] >= 0;
  const float share = r.always > 0 && live ? 1.f / (1.f + expf(-s[r.outputs])) : 0.f;
  const float total = route_choose(s, key, r.bias, r.correction, r.outputs, r.top, picked, 1);
  const int wide = r.top + r.always;
  for (int k = lane; k < wide; k += 32) {
    if (k >= r.top) {
      r.weight[(long long)row * wide + k] = share;
      continue;
    }
    const int e = picked[k];
    r.weight[(long long)row * wide + k] = live ? s[e] / (total + 1e-20f) : 0.f;
    r.choice[(long long)row * r.top + k] = live ? e : -1;
    r.rank[(long long)row * r.top + k] = live && e < r.experts ? atomicAdd(&r.count[e], 1) : -1;
  }
}

struct DispatchParams {
  const void* h;               // (rows, ld_h), `vecs` 16-byte pieces (or `d` elements) of a row are copied
  long long ld_h;
  void* xg;                    // (tiles * 128, ld_xg)
  long long ld_xg;
  const int *choice, *rank, *count;
  int* pos;                    // (rows, top + always): row of xg, -2 identity, -1 none
  int* tile_group;             // (tiles): expert, -1 = not used
  int rows, experts, top, always, tiles, d;
};

// E: an element, or 16 bytes of them.  One warp per row.
template <typename E>
__global__ void __launch_bounds__(256) moe_dispatch_kernel(const DispatchParams p) {
  pdl_sync();
  extern __shared__ int start[];             // [experts + always + 1]: first tile of every expert
  __shared__ int warp_sum[8];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int groups = p.experts + p.always;
  int carry = 0;
  for (int e0 = 0; e0 < groups; e0 += 256) {
    const int e = e0 + threadIdx.x;
    const int n = e < groups ? ((e < p.experts ? p.count[e] : p.rows) + ROUTE_TILE - 1) / ROUTE_TILE : 0;
    int x = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int y = __shfl_up_sync(0xffffffffu, x, o);
      if (lane >= o) x += y;
    }
    if (lane == 31) warp_sum[warp] = x;
    __syncthreads();
    int before = carry;
    for (int w = 0; w < 8; ++w) {
      if (w < warp) before += warp_sum[w];
      carry += warp_sum[w];
    }
    if (e < groups) start[e] = before + x - n;
    __syncthreads();
  }
  if (threadIdx.x == 0) start[groups] = carry;
  __syncthreads();
  if (blockIdx.x == 0) {
    for (int e = warp; e < groups; e += 8)
      for (int t = start[e] + lane; t < start[e + 1] && t < p.tiles; t += 32) p.tile_group[t] = e;
    for (int t = carry + threadIdx.x; t < p.tiles; t += 256) p.tile_group[t] = -1;
  }
  const int row = blockIdx.x * 8 + warp;
  if (row >= p.rows) return;
  const E* src = reinterpret_cast<const E*>(p.h) + row * p.ld_h;
  const int wide = p.top + p.always;
  for (int k0 = 0; k0 < wide; k0 += 32) {
    const int k = k0 + lane, n = min(32, wide - k0);
    int to = -1;
    if (k < wide) {
      const int e = p.choice[(long long)row * p.top + min(k, p.top - 1)];
      if (k >= p.top) to = e >= 0 ? start[p.experts + k - p.top] * ROUTE_TILE + row : -1;
      else if (e >= p.experts) to = -2;
      else if (e >= 0) to = start[e] * ROUTE_TILE + p.rank[(long long)row * p.top + k];
      if (to >= p.tiles * ROUTE_TILE) to = -1;
      p.pos[(long long)row * wide + k] = to;
    }
    for (int c0 = 0; c0 < p.d; c0 += 128) {
      E v[4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (c0 + i * 32 + lane < p.d) v[i] = src[c0 + i * 32 + lane];
      for (int j = 0; j < n; ++j) {
        const int at = __shfl_sync(0xffffffffu, to, j);
        if (at < 0) continue;
        E* dst = reinterpret_cast<E*>(p.xg) + at * p.ld_xg;
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (c0 + i * 32 + lane < p.d) dst[c0 + i * 32 + lane] = v[i];
      }
    }
  }
}

}  // namespace b200

using namespace b200;

static int route_params(RouteParams& p, const float* z, long long ld_z, const float* bias, const float* correction, const long long* slots, int* choice,
                        int* rank, float* weight, int* count, int rows, int experts, int outputs, int top, int always) {
  if (experts <= 0 || outputs < experts || top <= 0 || top > outputs || always < 0) return -10;
  p.z = z; p.ld_z = ld_z; p.bias = bias; p.correction = correction; p.slots = slots; p.choice = choice; p.rank = rank; p.weight = weight; p.count = count;
  p.rows = rows; p.experts = experts; p.outputs = outputs; p.top = top; p.always = always;
  return 0;
}

// `count` (experts ints) must be zero; identities are the outputs from `experts` on; with `always`, z has a column behind the outputs.
extern "C" int b200_moe_route(const float* z, long long ld_z, const float* bias, const float* correction, const long long* slots, int* choice,
                              int* rank, float* weight, int* count, int rows, int experts, int outputs, int top, int always, cudaStream_t st) {
  if (rows <= 0) return 0;
  RouteParams p;
  if (route_params(p, z, ld_z, bias, correction, slots, choice, rank, weight, count, rows, experts, outputs, top, always)) return -10;
  const size_t smem = (size_t)ROUTE_WARPS * 2 * outputs * 4 + 2ull * experts * 4 + (size_t)ROUTE_WARPS * ROUTE_ROWS * top * 8;
  if (smem > 200 * 1024) return -12;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return -3;
  launch_dep(moe_route_kernel, (unsigned)((rows + ROUTE_WARPS * ROUTE_ROWS - 1) / (ROUTE_WARPS * ROUTE_ROWS)), ROUTE_WARPS * 32, smem, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// The same for few rows, with the product: h (rows, d), w (columns, d), columns = outputs or one more; z (rows, ld_z) is written.
extern "C" int b200_moe_route_rows(const void* h, long long ld_h, const void* w, long long ld_w, int d, int columns, float* z, long long ld_z,
                                   const float* bias, const float* correction, const long long* slots, int* choice, int* rank, float* weight,
                                   int* count, int rows, int experts, int outputs, int top, int always, int f32, cudaStream_t st) {
  if (rows <= 0) return 0;
  RouteRowsParams p;
  if (route_params(p.r, z, ld_z, bias, correction, slots, choice, rank, weight, count, rows, experts, outputs, top, always)) return -10;
  if (d <= 0 || columns < outputs + (always > 0) || ld_z < columns) return -10;
  p.z = z; p.h = h; p.w = w; p.ld_h = ld_h; p.ld_w = ld_w; p.d = d; p.columns = columns;
  const size_t smem = (size_t)((columns + outputs + top + 3) / 4 * 4 + d) * 4;
  if (smem > 48 * 1024) return -12;
  const bool vec = d % 4 == 0 && ld_h % 4 == 0 && ld_w % 4 == 0 && ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(w)) & 15) == 0;
  if (f32) {
    if (vec) launch_dep(moe_route_rows_kernel<float, 4>, rows, 512, smem, st, p);
    else launch_dep(moe_route_rows_kernel<float, 1>, rows, 512, smem, st, p);
  } else {
    if (vec) launch_dep(moe_route_rows_kernel<__nv_bfloat16, 4>, rows, 512, smem, st, p);
    else launch_dep(moe_route_rows_kernel<__nv_bfloat16, 1>, rows, 512, smem, st, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// h (rows, d) of `elem`-byte elements, copied to its places in xg (tiles * 128, ld_xg).
extern "C" int b200_moe_dispatch(const void* h, long long ld_h, void* xg, long long ld_xg, const int* choice, const int* rank,
                                 const int* count, int* pos, int* tile_group, int rows, int experts, int top, int always, int tiles, int d,
                                 int elem, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (experts <= 0 || always < 0 || experts + always > 4096 || top <= 0 || tiles <= 0 || d <= 0 || (elem != 2 && elem != 4)) return -10;
  DispatchParams p;
  p.h = h; p.ld_h = ld_h; p.xg = xg; p.ld_xg = ld_xg; p.choice = choice; p.rank = rank; p.count = count; p.pos = pos;
  p.tile_group = tile_group; p.rows = rows; p.experts = experts; p.top = top; p.always = always; p.tiles = tiles; p.d = d;
  const unsigned grid = (unsigned)((rows + 7) / 8);
  const size_t smem = (experts + always + 1) * sizeof(int);
  const int per = 16 / elem;
  if (d % per == 0 && ld_h % per == 0 && ld_xg % per == 0 && ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(xg)) & 15) == 0) {
    p.d = d / per; p.ld_h = ld_h / per; p.ld_xg = ld_xg / per;
    launch_dep(moe_dispatch_kernel<uint4>, grid, 256, smem, st, p);
  } else if (elem == 2) {
    launch_dep(moe_dispatch_kernel<uint16_t>, grid, 256, smem, st, p);
  } else {
    launch_dep(moe_dispatch_kernel<uint32_t>, grid, 256, smem, st, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
