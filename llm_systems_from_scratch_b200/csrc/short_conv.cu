// Short causal convolution over time, a filter of `taps` weights per channel:
//     y_t[c] = act(sum_j w[j][c] u_(t - taps + 1 + j)[c])
// with zeros in front of a sequence.  What a sequence's next step needs of the earlier ones lives in a ring of `taps` rows in its state
// slot: position t in row t mod taps.  A step of single rows reads its taps - 1 predecessors there and leaves its own input in the row
// that none of them uses; portions leave their last rows by short_conv_carry, after every block of the convolution has read the ring.
// Either the result is written as a matrix, or it goes where grouped attention wants it: queries, times a number per head, into padded
// vectors; keys and values into the cache, the values mixed with those that an earlier layer has cached for the same token.
#include "grouped_attention.cuh"

namespace b200 {

struct ConvParams {
  const void* u;               // (rows, ld_u)
  long long ld_u;
  const void* w;               // (taps, channels)
  void* ring;                  // (num_slots, taps, channels)
  const int* state_slots;      // per sequence; negative = padding
  const int* row_seq;          // sequence of a row, less seq0; null: row i is sequence i
  const int* cu;               // (seqs + 1) rows of each sequence; null: one row each
  const int* positions;        // per row
  int seq0, seqs, rows, channels, taps, num_slots;
  void* y;                     // plain: (rows, ld_y)
  long long ld_y;
  int silu;
  // attention: channels are q (heads, dim) | k (kv_heads, dim) | v (kv_heads, vdim)
  void *q, *cache;
  const long long* slots;
  const float* temp;           // (heads)
  const void* first;           // cache of the earlier layer whose values are mixed in, or null
  long long first_width, first_off, cache_slots;
  int first_pitch;
  float mix;
  GroupedShape s;
  uint32_t* status;
};

template <int VEC, typename T>
__device__ __forceinline__ void conv_load(const T* p, float (&f)[VEC]) {
  if constexpr (VEC == 8) unpack(load_piece(p), f);
  else f[0] = to_f(*p);
}
template <int VEC, typename T>
__device__ __forceinline__ void conv_store(T* p, const float (&f)[VEC]) {
  if constexpr (VEC == 8) store8(p, f);
  else from_f(*p, f[0]);
}

__device__ __forceinline__ float conv_silu(float y, float) { return y / (1.f + expf(-y)); }                           // fp32 activations
__device__ __forceinline__ float conv_silu(float y, __nv_bfloat16) { return __fdividef(y, 1.f + __expf(-y)); }

// Where VEC channels from c on go (attention), and what becomes of them.
template <typename T, int VEC>
struct ConvTarget {
  bool query, key;
  int head, e, len, pitch;
  float temp;
  __device__ __forceinline__ ConvTarget(const ConvParams& p, int c, bool attend) {
    if (!attend) return;
    const GroupedShape& s = p.s;
    const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim;
    query = c < nq;
    key = !query && c < nq + nk;
    const int at = query ? c : (key ? c - nq : c - nq - nk);
    len = query || key ? s.dim : s.vdim;
    head = at / len;
    e = at - head * len;
    pitch = query ? s.qp : (key ? s.kp : s.vp);
    temp = query ? p.temp[head] : 1.f;
  }
  // v_first of the same token, where values are mixed
  __device__ __forceinline__ const T* first(const ConvParams& p, long long to) const {
    return reinterpret_cast<const T*>(p.first) + to * p.first_width + p.first_off + head * p.first_pitch + e;
  }
  __device__ __forceinline__ bool mixes(const ConvParams& p) const { return !query && !key && p.first != nullptr; }
  __device__ __forceinline__ void put(const ConvParams& p, int row, long long to, const float (&v1)[VEC], float (&y)[VEC]) const {
    const GroupedShape& s = p.s;
    T* dst;
    if (query) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] *= temp;
      dst = reinterpret_cast<T*>(p.q) + ((long long)row * s.heads + head) * s.qp;
    } else {
      if (mixes(p)) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] = (1.f - p.mix) * y[i] + p.mix * v1[i];
      }
      dst = reinterpret_cast<T*>(p.cache) + to * (long long)(s.kv_heads * (s.kp + s.vp)) + (key ? head * s.kp : s.kv_heads * s.kp + head * s.vp);
    }
    conv_store<VEC>(dst + e, y);
    if (e + VEC == len) {                                // the pad behind the vector
      float z[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) z[i] = 0.f;
      for (int k = len; k + VEC <= pitch; k += VEC) conv_store<VEC>(dst + k, z);
    }
  }
};

// y = the convolution of VEC channels of one row; false where an index is bad.
template <typename T, int VEC>
__device__ __forceinline__ bool conv_row(const ConvParams& p, int c, int row, float (&y)[VEC]) {
  const int taps = p.taps;
  const T* u = reinterpret_cast<const T*>(p.u) + (long long)row * p.ld_u + c;
  const T* w = reinterpret_cast<const T*>(p.w) + c;
  float now[VEC], g[VEC];
  conv_load<VEC>(u, now);
  conv_load<VEC>(w + (long long)(taps - 1) * p.channels, g);
  const int seq = p.row_seq != nullptr ? p.row_seq[row] - p.seq0 : row, pos = p.positions[row];
  if ((unsigned)seq >= (unsigned)p.seqs) {
    report_bad_arg(p.status, 30);
    return false;
  }
  const int first = p.cu != nullptr ? p.cu[seq] : row;
  int slot = p.state_slots[seq];
  if (slot >= p.num_slots) {
    report_bad_arg(p.status, 31);
    slot = -1;
  }
  T* ring = reinterpret_cast<T*>(p.ring) + (long long)max(slot, 0) * taps * p.channels + c;
#pragma unroll
  for (int i = 0; i < VEC; ++i) y[i] = g[i] * now[i];
#pragma unroll 3
  for (int d = 1; d < taps; ++d) {
    float f[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) f[i] = 0.f;
    if (row - d >= first) conv_load<VEC>(u - d * p.ld_u, f);
    else if (pos >= d && slot >= 0) conv_load<VEC>(ring + (long long)((pos - d) % taps) * p.channels, f);
    conv_load<VEC>(w + (long long)(taps - 1 - d) * p.channels, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) y[i] = fmaf(g[i], f[i], y[i]);
  }
  if (p.cu == nullptr && slot >= 0) conv_store<VEC>(ring + (long long)(pos % taps) * p.channels, now);
  return true;
}

// What becomes of a row's y: stored, or sent where attention wants it (v1: the values to mix in).
template <typename T, int VEC, bool ATTEND>
__device__ __forceinline__ void conv_finish(const ConvParams& p, const ConvTarget<T, VEC>& at, int c, int row, long long to, const float (&v1)[VEC],
                                            float (&y)[VEC]) {
  if constexpr (ATTEND) {
    if (!at.query && to < 0) return;                     // padding row of the batch
    if (!at.query && to >= p.cache_slots) {
      report_bad_arg(p.status, 32);
      return;
    }
    at.put(p, row, to, v1, y);
  } else {
    if (p.silu) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] = conv_silu(y[i], T());
    }
    conv_store<VEC>(reinterpret_cast<T*>(p.y) + (long long)row * p.ld_y + c, y);
  }
}

// One row per thread and piece of VEC channels: any number of taps, single rows (which leave their input in the ring) and portions.
template <typename T, int VEC, bool ATTEND>
__global__ void __launch_bounds__(256) short_conv_kernel(const ConvParams p) {
  pdl_sync();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC, row = blockIdx.x;
  if (c >= p.channels) return;
  const long long to = ATTEND ? p.slots[row] : 0;
  const ConvTarget<T, VEC> at(p, c, ATTEND);
  float y[VEC], v1[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) v1[i] = 0.f;
  if (ATTEND && at.mixes(p) && to >= 0 && to < p.cache_slots) conv_load<VEC>(at.first(p, to), v1);
  if (conv_row<T, VEC>(p, c, row, y)) conv_finish<T, VEC, ATTEND>(p, at, c, row, to, v1, y);
}

template <bool ATTEND>
constexpr int CONV_RUN = ATTEND ? 4 : 8;

// CONV_RUN rows of portions per thread and piece of 8 channels: every row is requested once, before the first is worked on, and stays in
// registers for the rows behind it.  Where a sequence ends among them, they are taken one by one.
template <typename T, int TAPS, bool ATTEND>
__global__ void __launch_bounds__(256) short_conv_run_kernel(const ConvParams p) {
  pdl_sync();
  constexpr int RUN = CONV_RUN<ATTEND>, H = TAPS - 1;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8, r0 = blockIdx.x * RUN, n = min(RUN, p.rows - r0);
  if (c >= p.channels) return;
  const T* u = reinterpret_cast<const T*>(p.u) + c;
  Piece<T> in[H + RUN], filter[TAPS], mixed[ATTEND ? RUN : 1];
  long long to[RUN];
  const ConvTarget<T, 8> at(p, c, ATTEND);
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    if (i < n) in[H + i] = load_piece(u + (long long)(r0 + i) * p.ld_u);
    to[i] = ATTEND && i < n ? p.slots[r0 + i] : -1;
  }
#pragma unroll
  for (int j = 0; j < TAPS; ++j) filter[j] = load_piece(reinterpret_cast<const T*>(p.w) + (long long)j * p.channels + c);
  const int seq = p.row_seq[r0] - p.seq0;
  if (seq == p.row_seq[r0 + n - 1] - p.seq0 && (unsigned)seq < (unsigned)p.seqs) {
    const int first = p.cu[seq], pos = p.positions[r0];
    int slot = p.state_slots[seq];
    if (slot >= p.num_slots) {
      report_bad_arg(p.status, 31);
      slot = -1;
    }
    const T* ring = reinterpret_cast<const T*>(p.ring) + (long long)max(slot, 0) * TAPS * p.channels + c;
#pragma unroll
    for (int d = 1; d <= H; ++d) {
#pragma unroll
      for (int k = 0; k < (int)sizeof(T) / 2; ++k) in[H - d].v[k] = make_uint4(0, 0, 0, 0);
      if (r0 - d >= first) in[H - d] = load_piece(u + (long long)(r0 - d) * p.ld_u);
      else if (pos >= d && slot >= 0) in[H - d] = load_piece(ring + (long long)((pos - d) % TAPS) * p.channels);
    }
    if constexpr (ATTEND) {
      if (at.mixes(p)) {
#pragma unroll
        for (int i = 0; i < RUN; ++i)
          if (to[i] >= 0 && to[i] < p.cache_slots) mixed[i] = load_piece(at.first(p, to[i]));
      }
    }
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
      if (i >= n) break;
      float y[8], g[8], f[8], v1[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) y[k] = v1[k] = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        unpack(filter[j], g);
        unpack(in[i + j], f);
#pragma unroll
        for (int k = 0; k < 8; ++k) y[k] = fmaf(g[k], f[k], y[k]);
      }
      if constexpr (ATTEND) {
        if (at.mixes(p) && to[i] >= 0 && to[i] < p.cache_slots) unpack(mixed[i], v1);
      }
      conv_finish<T, 8, ATTEND>(p, at, c, r0 + i, to[i], v1, y);
    }
    return;
  }
  for (int i = 0; i < n; ++i) {
    float y[8], v1[8];
    const long long line = ATTEND ? p.slots[r0 + i] : 0;
#pragma unroll
    for (int k = 0; k < 8; ++k) v1[k] = 0.f;
    if (ATTEND && at.mixes(p) && line >= 0 && line < p.cache_slots) conv_load<8>(at.first(p, line), v1);
    if (conv_row<T, 8>(p, c, r0 + i, y)) conv_finish<T, 8, ATTEND>(p, at, c, r0 + i, line, v1, y);
  }
}

// The last taps - 1 rows of every portion into its ring.
template <typename T>
__global__ void __launch_bounds__(256) short_conv_carry_kernel(const ConvParams p) {
  pdl_sync();
  const int seq = blockIdx.x, slot = p.state_slots[seq];
  if (slot < 0 || slot >= p.num_slots) return;
  const int row0 = p.cu[seq], row1 = p.cu[seq + 1];
  T* ring = reinterpret_cast<T*>(p.ring) + (long long)slot * p.taps * p.channels;
  for (int d = 1; d < p.taps && row1 - d >= row0; ++d) {
    const int row = row1 - d;
    const T* u = reinterpret_cast<const T*>(p.u) + (long long)row * p.ld_u;
    T* to = ring + (long long)(p.positions[row] % p.taps) * p.channels;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < p.channels; c += gridDim.y * blockDim.x) to[c] = u[c];
  }
}

template <typename T, bool ATTEND>
static void launch_conv(const ConvParams& p, bool vec, cudaStream_t st) {
  const int pieces = p.channels / (vec ? 8 : 1);
  const int threads = pieces >= 256 ? 256 : (pieces + 31) / 32 * 32;
  const unsigned gy = (pieces + threads - 1) / threads;
  const bool run = vec && p.cu != nullptr && p.taps >= 2 && p.taps <= 4 && (long long)p.rows * pieces >= 148ll * 2048 * 2;
  const dim3 grid(run ? (p.rows + CONV_RUN<ATTEND> - 1) / CONV_RUN<ATTEND> : p.rows, gy);
  if (!vec) launch_dep(short_conv_kernel<T, 1, ATTEND>, grid, threads, 0, st, p);
  else if (!run) launch_dep(short_conv_kernel<T, 8, ATTEND>, grid, threads, 0, st, p);
  else if (p.taps == 2) launch_dep(short_conv_run_kernel<T, 2, ATTEND>, grid, threads, 0, st, p);
  else if (p.taps == 3) launch_dep(short_conv_run_kernel<T, 3, ATTEND>, grid, threads, 0, st, p);
  else launch_dep(short_conv_run_kernel<T, 4, ATTEND>, grid, threads, 0, st, p);
  if (p.cu != nullptr && p.taps > 1)
    launch_dep(short_conv_carry_kernel<T>, dim3(p.seqs, p.channels >= 1024 ? 4 : 1), 256, 0, st, p);
}

}  // namespace b200

using namespace b200;

// A convolution's input, state and rows, passed by pointer through the C interface: the field order is part of it.
struct ConvInput {
  const void* u;
  const void* w;
  void* ring;
  const int *state_slots, *row_seq, *cu, *positions;
  long long ld_u;
  int seq0, seqs, rows, channels, taps, num_slots;
};

static int conv_params(ConvParams& p, const ConvInput& in, uint32_t* status) {
  if (in.channels <= 0 || in.taps <= 0 || in.seqs <= 0 || in.num_slots <= 0 || in.u == nullptr || in.w == nullptr || in.ring == nullptr ||
      (in.cu == nullptr && in.seqs != in.rows) || (in.cu != nullptr && in.row_seq == nullptr))
    return -10;
  p = {};
  p.u = in.u; p.ld_u = in.ld_u; p.w = in.w; p.ring = in.ring; p.state_slots = in.state_slots; p.row_seq = in.row_seq; p.cu = in.cu;
  p.positions = in.positions; p.seq0 = in.seq0; p.seqs = in.seqs; p.rows = in.rows; p.channels = in.channels; p.taps = in.taps;
  p.num_slots = in.num_slots; p.status = status;
  return 0;
}
static bool conv_vec(const ConvInput& in, uintptr_t more) {
  return in.channels % 8 == 0 && in.ld_u % 8 == 0 &&
         ((reinterpret_cast<uintptr_t>(in.u) | reinterpret_cast<uintptr_t>(in.w) | reinterpret_cast<uintptr_t>(in.ring) | more) & 15) == 0;
}

// y (rows, ld_y) = the convolution, with silu if asked for.
extern "C" int b200_short_conv(const ConvInput* in, void* y, long long ld_y, int silu, int f32, uint32_t* status, cudaStream_t st) {
  if (in->rows <= 0) return 0;
  ConvParams p;
  if (conv_params(p, *in, status) || y == nullptr) return -10;
  p.y = y; p.ld_y = ld_y; p.silu = silu;
  const bool vec = conv_vec(*in, reinterpret_cast<uintptr_t>(y)) && ld_y % 8 == 0;
  if (f32) launch_conv<float, false>(p, vec, st);
  else launch_conv<__nv_bfloat16, false>(p, vec, st);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// The convolution of q | k | v of grouped attention: q (rows, heads * qp), times temp (heads); keys and values into `cache`.  first: cache
// (same pages, lines of first_width elements, a head's values at first_off + head * first_pitch) whose values are mixed in with weight
// `mix`, or null.
extern "C" int b200_short_conv_attend(const ConvInput* in, void* q, void* cache, const long long* slots, long long cache_slots,
                                      const float* temp, const void* first, long long first_width, long long first_off, int first_pitch,
                                      float mix, const GroupedShape* s, int f32, uint32_t* status, cudaStream_t st) {
  if (in->rows <= 0) return 0;
  ConvParams p;
  if (conv_params(p, *in, status) || !shape_ok(*s) || s->maps != 1 || q == nullptr || cache == nullptr || temp == nullptr ||
      in->channels != s->heads * s->dim + s->kv_heads * (s->dim + s->vdim))
    return -10;
  p.q = q; p.cache = cache; p.slots = slots; p.cache_slots = cache_slots; p.temp = temp; p.first = first; p.first_width = first_width;
  p.first_off = first_off; p.first_pitch = first_pitch; p.mix = mix; p.s = *s;
  const bool vec = conv_vec(*in, reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(first)) &&
                   s->dim % 8 == 0 && s->vdim % 8 == 0 && first_width % 8 == 0 && first_off % 8 == 0 && first_pitch % 8 == 0;
  if (f32) launch_conv<float, true>(p, vec, st);
  else launch_conv<__nv_bfloat16, true>(p, vec, st);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
