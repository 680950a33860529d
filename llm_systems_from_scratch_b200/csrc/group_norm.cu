// Passes over the fp32 residual stream of designs with norms in groups, gated sublayers and norms on both sides of them:
//     u = sublayer output * sigmoid(gate)         elementwise, the gate's pre-activations come with the sublayer's input products
//     x = x + group_norm(u) * w_post
//     h = group_norm(x) * w                       input of the next sublayer
// in one pass, one block per row.  group_norm: equal consecutive parts of a row, each over its own root mean square.  A sublayer's output is
// a matrix, or the weighted outputs of the experts a row has chosen.  The first pass starts the row instead: an embedding times a scale
// plus a row of a table that belongs to the pair (previous token, token); the previous token is part of a sequence's state.
#include "typed.cuh"

namespace b200 {

struct GroupStepParams {
  float* x;                    // (rows, d) fp32
  int rows, x_rows, d, groups;
  float eps;
  // start
  const long long* tokens;     // null: no start
  const void *embed, *bigram;  // (vocab, d), (buckets + 1, d) or null
  int vocab, buckets;
  long long mul_prev, mul_cur;
  float scale;
  int* prev;                   // (num_slots): last token of a sequence
  const int *state_slots, *row_seq, *positions;
  int num_slots, n_single;     // rows below n_single are their sequence's only row of the step: they keep their token here
  // sublayer
  const void* y;               // (rows, ld_y), or (y_rows, ld_y) with ypos; null: none
  long long ld_y;
  const int* ypos;             // (rows, ytop): row of y, negative: none
  const float* yweight;        // (rows, ytop)
  int ytop, y_rows;
  const void* gate;            // (rows, ld_gate)
  long long ld_gate;
  const void* w_post;
  // next input
  const long long* row_index;  // optional: h[i] is of row row_index[i]; x is not written
  const void* w;               // null: no h
  void* h;
  long long ld_h;
  uint32_t* status;
};

template <int VEC, typename T>
__device__ __forceinline__ void gs_load(const T* p, float (&f)[VEC]) {
  if constexpr (VEC == 8) unpack(load_piece(p), f);
  else load_vec<VEC>(p, f);
}
template <int VEC, typename T>
__device__ __forceinline__ void gs_store(T* p, const float (&f)[VEC]) {
  if constexpr (VEC == 8) store8(p, f);
  else store_vec<VEC>(p, f);
}
template <typename T>
__device__ __forceinline__ float gs_gated(float u, float g) {
  if constexpr (sizeof(T) == 4) return u / (1.f + expf(-g));
  else return __fdividef(u, 1.f + __expf(-g));
}

// A thread holds KEEP pieces of VEC columns: columns c0 + j * step.  1 << seg lanes next to each other are inside one group.
template <typename T, int VEC, int KEEP>
__global__ void __launch_bounds__(512) group_step_kernel(const GroupStepParams p, const int seg) {
  pdl_sync();
  extern __shared__ float gsum[];                        // [2][d / (VEC << seg)] sums of squares
  const int row = blockIdx.x, step = blockDim.x * VEC, c0 = threadIdx.x * VEC;
  constexpr int SHIFT = VEC == 8 ? 3 : (VEC == 4 ? 2 : 0);
  const int lanes = 1 << seg, size = p.d / p.groups, per_group = size >> (seg + SHIFT), segs = p.d >> (seg + SHIFT);
  const float share = 1.f / (float)size;
  long long src = row;
  if (p.row_index != nullptr) {
    src = p.row_index[row];
    if (src < 0 || src >= p.x_rows) {
      if (threadIdx.x == 0) report_bad_arg(p.status, 40);
      src = 0;
    }
  }
  float* xr = p.x + src * p.d;
  // everything that is read in any case is requested first
  float x[KEEP][VEC];
  Raw<T, VEC> gate[KEEP], post[KEEP], w[KEEP], raw[KEEP];
  auto request = [&](const T* from, Raw<T, VEC> (&to)[KEEP]) __attribute__((always_inline)) {
#pragma unroll
    for (int j = 0; j < KEEP; ++j)
      if (c0 + j * step < p.d) to[j] = *reinterpret_cast<const Raw<T, VEC>*>(from + c0 + j * step);
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[j][i] = 0.f;
    if (p.tokens == nullptr && c0 + j * step < p.d) gs_load<VEC>(xr + c0 + j * step, x[j]);
  }
  if (p.y != nullptr) {
    request(reinterpret_cast<const T*>(p.gate) + src * p.ld_gate, gate);
    if (p.ypos == nullptr) request(reinterpret_cast<const T*>(p.y) + src * p.ld_y, raw);
    request(reinterpret_cast<const T*>(p.w_post), post);
  }
  if (p.h != nullptr) request(reinterpret_cast<const T*>(p.w), w);
  int first[KEEP];                                       // first sum of a piece's group
#pragma unroll
  for (int j = 0; j < KEEP; ++j) first[j] = (c0 + j * step) / size * per_group;
  // norm of the thread's pieces f in place: f / rms of the group * weight
  auto norm = [&](float (&f)[KEEP][VEC], const Raw<T, VEC> (&weight)[KEEP], float* sums) __attribute__((always_inline)) {
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(f[j][i], f[j][i], ss);
      for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const int c = c0 + j * step;
      if (c < p.d && (threadIdx.x & (lanes - 1)) == 0) sums[c >> (seg + SHIFT)] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      if (c0 + j * step >= p.d) break;
      float ss = 0.f;
      for (int k = 0; k < per_group; ++k) ss += sums[first[j] + k];
      const float r = rsqrtf(fmaf(ss, share, p.eps));
      float g[VEC];
      gs_load<VEC>(weight[j].v, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) f[j][i] *= r * g[i];
    }
  };
  if (p.tokens != nullptr) {
    long long tok = p.tokens[row];
    if (tok < 0 || tok >= p.vocab) {
      if (threadIdx.x == 0) report_bad_arg(p.status, 41);
      tok = 0;
    }
    const T* er = reinterpret_cast<const T*>(p.embed) + tok * p.d;
    const T* br = nullptr;
    if (p.bigram != nullptr) {
      const int seq = p.row_seq[row], slot = p.state_slots[seq];
      long long pair = p.buckets;
      if (p.positions[row] > 0) {
        const bool inside = row > 0 && p.row_seq[row - 1] == seq;
        const long long before = inside ? p.tokens[row - 1] : (slot >= 0 && slot < p.num_slots ? p.prev[slot] : 0);
        pair = (before * p.mul_prev + tok * p.mul_cur) % p.buckets;
        if (pair < 0) pair += p.buckets;
      }
      br = reinterpret_cast<const T*>(p.bigram) + pair * p.d;
      __syncthreads();                                   // everybody has read the previous token
      if (row < p.n_single && threadIdx.x == 0 && slot >= 0 && slot < p.num_slots) p.prev[slot] = (int)tok;
    }
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      const int c = c0 + j * step;
      if (c >= p.d) break;
      float b[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) b[i] = 0.f;
      gs_load<VEC>(er + c, x[j]);
      if (br != nullptr) gs_load<VEC>(br + c, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[j][i] = fmaf(x[j][i], p.scale, b[i]);
      gs_store<VEC>(xr + c, x[j]);
    }
  }
  if (p.y != nullptr) {
    float u[KEEP][VEC];
#pragma unroll
    for (int j = 0; j < KEEP; ++j)
#pragma unroll
      for (int i = 0; i < VEC; ++i) u[j][i] = 0.f;
    if (p.ypos == nullptr) {
#pragma unroll
      for (int j = 0; j < KEEP; ++j)
        if (c0 + j * step < p.d) gs_load<VEC>(raw[j].v, u[j]);
    } else {
#pragma unroll 2
      for (int k = 0; k < p.ytop; ++k) {
        const int pos = p.ypos[src * p.ytop + k];
        if (pos < 0 || pos >= p.y_rows) continue;        // a padding row of the batch
        const float a = p.yweight[src * p.ytop + k];
        request(reinterpret_cast<const T*>(p.y) + (long long)pos * p.ld_y, raw);
#pragma unroll
        for (int j = 0; j < KEEP; ++j)
          if (c0 + j * step < p.d) {
            float f[VEC];
            gs_load<VEC>(raw[j].v, f);
#pragma unroll
            for (int i = 0; i < VEC; ++i) u[j][i] = fmaf(a, f[i], u[j][i]);
          }
      }
    }
#pragma unroll
    for (int j = 0; j < KEEP; ++j)
      if (c0 + j * step < p.d) {
        float g[VEC];
        gs_load<VEC>(gate[j].v, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[j][i] = gs_gated<T>(u[j][i], g[i]);
      }
    norm(u, post, gsum);
#pragma unroll
    for (int j = 0; j < KEEP; ++j)
      if (c0 + j * step < p.d) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[j][i] += u[j][i];
        if (p.row_index == nullptr) gs_store<VEC>(xr + c0 + j * step, x[j]);
      }
  }
  if (p.h == nullptr) return;
  norm(x, w, gsum + segs);
  T* hr = reinterpret_cast<T*>(p.h) + (long long)row * p.ld_h;
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if (c0 + j * step < p.d) gs_store<VEC>(hr + c0 + j * step, x[j]);
}

// The last token of every portion into its sequence's state.
__global__ void carry_tokens_kernel(const long long* tokens, const int* cu, const int* state_slots, int* prev, int seqs, int num_slots) {
  pdl_sync();
  const int seq = blockIdx.x * blockDim.x + threadIdx.x;
  if (seq >= seqs) return;
  const int slot = state_slots[seq];
  if (slot >= 0 && slot < num_slots && cu[seq + 1] > cu[seq]) prev[slot] = (int)tokens[cu[seq + 1] - 1];
}

template <typename T, int VEC>
static int launch_group_step(const GroupStepParams& p, cudaStream_t st) {
  const int pieces = p.d / VEC, size = p.d / p.groups;
  int seg = 0;
  while (seg < 5 && size % ((2 << seg) * VEC) == 0) ++seg;
  const int want = p.rows >= 148 * 8 && VEC < 8 ? (pieces + 1) / 2 : pieces;      // many rows share an SM, few have all of its threads
  int threads = (want + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const int keep = (pieces + threads - 1) / threads;
  const size_t smem = 2ull * (p.d / (VEC << seg)) * sizeof(float);
  if (smem > 48 * 1024) return -12;
  if (keep <= 1) launch_dep(group_step_kernel<T, VEC, 1>, p.rows, threads, smem, st, p, seg);
  else if (keep <= 2) launch_dep(group_step_kernel<T, VEC, 2>, p.rows, threads, smem, st, p, seg);
  else if (keep <= 4) launch_dep(group_step_kernel<T, VEC, 4>, p.rows, threads, smem, st, p, seg);
  else if (VEC < 8 && keep <= 16) launch_dep(group_step_kernel<T, VEC < 8 ? VEC : 4, 16>, p.rows, threads, smem, st, p, seg);
  else return -12;
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace b200

using namespace b200;

// Passed by pointer through the C interface: the field order is part of it.
struct GroupStart {
  const long long* tokens;
  const void *embed, *bigram;
  int* prev;
  const int *state_slots, *row_seq, *positions, *cu;     // cu: rows of the portions, counted from row n_single; null without portions
  long long mul_prev, mul_cur;
  int vocab, buckets, num_slots, n_single, portions;
  float scale;
};
struct GroupSublayer {
  const void *y, *gate, *w_post;
  const int* ypos;
  const float* yweight;
  long long ld_y, ld_gate;
  int ytop, y_rows;
};

extern "C" int b200_group_step(float* x, const GroupStart* start, const GroupSublayer* sub, const long long* row_index, const void* w, void* h,
                               long long ld_h, float eps, int rows, int x_rows, int d, int groups, int f32, uint32_t* status,
                               cudaStream_t st) {
  if (rows <= 0) return 0;
  if (x == nullptr || d <= 0 || groups <= 0 || d % groups || (h != nullptr && w == nullptr) || (start != nullptr && row_index != nullptr)) return -10;
  GroupStepParams p = {};
  p.x = x; p.rows = rows; p.x_rows = x_rows; p.d = d; p.groups = groups; p.eps = eps; p.row_index = row_index; p.w = w; p.h = h; p.ld_h = ld_h;
  p.status = status;
  if (start != nullptr) {
    if (start->embed == nullptr || (start->bigram != nullptr && (start->prev == nullptr || start->buckets <= 0))) return -10;
    p.tokens = start->tokens; p.embed = start->embed; p.bigram = start->bigram; p.vocab = start->vocab; p.buckets = start->buckets;
    p.mul_prev = start->mul_prev; p.mul_cur = start->mul_cur; p.scale = start->scale; p.prev = start->prev;
    p.state_slots = start->state_slots; p.row_seq = start->row_seq; p.positions = start->positions; p.num_slots = start->num_slots;
    p.n_single = start->n_single;
  }
  if (sub != nullptr) {
    if (sub->y == nullptr || sub->gate == nullptr || sub->w_post == nullptr || (sub->ypos != nullptr && sub->yweight == nullptr)) return -10;
    p.y = sub->y; p.ld_y = sub->ld_y; p.gate = sub->gate; p.ld_gate = sub->ld_gate; p.w_post = sub->w_post; p.ypos = sub->ypos;
    p.yweight = sub->yweight; p.ytop = sub->ytop; p.y_rows = sub->y_rows;
  }
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(p.embed) | reinterpret_cast<uintptr_t>(p.bigram) |
                         reinterpret_cast<uintptr_t>(p.y) | reinterpret_cast<uintptr_t>(p.gate) | reinterpret_cast<uintptr_t>(p.w_post) |
                         reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(h);
  const bool vec = (d / groups) % 4 == 0 && (p.ld_y | p.ld_gate | ld_h) % 4 == 0 && (ptrs & 15) == 0;
  const bool wide = vec && (d / groups) % 8 == 0 && (p.ld_y | p.ld_gate | ld_h) % 8 == 0 && d <= 8192 && rows >= 148 * 4;
  int r;
  if (f32) r = vec ? launch_group_step<float, 4>(p, st) : launch_group_step<float, 1>(p, st);
  else if (wide) r = launch_group_step<__nv_bfloat16, 8>(p, st);
  else r = vec ? launch_group_step<__nv_bfloat16, 4>(p, st) : launch_group_step<__nv_bfloat16, 1>(p, st);
  if (r == 0 && start != nullptr && start->bigram != nullptr && start->portions > 0) {
    launch_dep(carry_tokens_kernel, (start->portions + 127) / 128, 128, 0, st, start->tokens + start->n_single, start->cu,
               start->state_slots + start->n_single, start->prev, start->portions, start->num_slots);
    r = cudaGetLastError() == cudaSuccess ? 0 : -4;
  }
  return r;
}
