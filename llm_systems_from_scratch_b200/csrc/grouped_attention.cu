// Softmax attention of grouped heads over a paged cache: query head h reads key/value head h / (heads / kv_heads), under a
// sliding window (position i sees the `window` positions up to and including i, and the first `keep` positions of the sequence) or inside
// chunks of `window` positions counted from the sequence's first, with optional parts: scores capped softly (cap tanh(score / cap)), a bias
// per distance from a table or linear in it, a sink per head (exp(sink) joins the softmax's denominator) and, for differential attention, two maps per head over the same values:
//     o = a_1 - difference * a_2,   o <- o / rms(o) * out_scale
// and an optional gate, o * sigmoid(g), per element or per head.  This file: norm, rotation and append; the general kernel (any size, bf16 or fp32);
// decode on mma.sync.  Portions of prompts: grouped_prefill.cu.
//
// Cache row of a token: kv_heads x maps keys of kp elements, then kv_heads values of vp elements (kp, vp: dim, vdim rounded
// up to 8, zero padded).  Query rows: heads x maps vectors of qp elements, zero padded.
#include "grouped_attention.cuh"

namespace b200 {

// ------------------------------------------------------------------------------------------- norm, rotation, append
struct GroupedPrepParams {
  const void* proj;            // (rows, ld): q (heads, maps, dim) | k (kv_heads, maps, dim) | v (kv_heads, vdim) | ...
  long long ld;
  void* q;                     // (rows, heads * maps * qp)
  void* cache;
  const void *wq, *wk;         // (dim); wk null: the layer has no keys and values of its own
  const float* cos_sin;        // (2, ctx, rot / 2)
  const int* positions;
  const long long* slots;
  int rows, heads, kv_heads, maps, dim, vdim, qp, kp, vp, rot, ctx;
  long long num_slots;
  float eps;
  uint32_t* status;
};

// One warp per vector: a query or key of one head and map (norm, rotation), or a value (copied).
template <typename T, int VEC>
__global__ void __launch_bounds__(256) grouped_prep_kernel(const GroupedPrepParams p) {
  pdl_sync();
  const int lane = threadIdx.x & 31;
  const int nq = p.heads * p.maps, nk = p.wk != nullptr ? p.kv_heads * p.maps : 0, nv = p.wk != nullptr ? p.kv_heads : 0;
  const int per = nq + nk + nv;
  const long long item = blockIdx.x * (long long)(blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= (long long)p.rows * per) return;
  const int row = (int)(item / per), j = (int)(item - (long long)row * per);
  const T* pr = reinterpret_cast<const T*>(p.proj) + (long long)row * p.ld;
  T* dst;
  const T* src;
  const T* w = nullptr;
  int len = p.dim, pad;
  if (j < nq) {
    src = pr + j * p.dim;
    dst = reinterpret_cast<T*>(p.q) + ((long long)row * nq + j) * p.qp;
    w = reinterpret_cast<const T*>(p.wq);
    pad = p.qp;
  } else {
    const long long slot = p.slots[row];
    if (slot < 0) return;                       // padding row of the batch
    if (slot >= p.num_slots) {
      if (lane == 0) report_bad_arg(p.status, 13);
      return;
    }
    T* cr = reinterpret_cast<T*>(p.cache) + slot * ((long long)p.kv_heads * (p.maps * p.kp + p.vp));
    if (j < nq + nk) {
      src = pr + j * p.dim;                     // the keys follow the queries
      dst = cr + (j - nq) * p.kp;
      w = reinterpret_cast<const T*>(p.wk);
      pad = p.kp;
    } else {
      const int g = j - nq - nk;
      src = pr + (nq + nk) * p.dim + g * p.vdim;
      dst = cr + nk * p.kp + g * p.vp;
      len = p.vdim;
      pad = p.vp;
    }
  }
  float r = 1.f;
  int pos = 0;
  if (w != nullptr) {
    float ss = 0.f;
    for (int c = lane * VEC; c < len; c += 32 * VEC) {
      float f[VEC];
      load_vec<VEC>(src + c, f);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss += f[i] * f[i];
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    r = rsqrtf(ss / (float)len + p.eps);
    pos = p.positions[row];
    if (p.rot > 0 && (pos < 0 || pos >= p.ctx)) {
      if (lane == 0) report_bad_arg(p.status, 14);
      pos = 0;
    }
  }
  const int half = p.rot / 2;
  for (int c = lane * VEC; c < pad; c += 32 * VEC) {
    float f[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) f[i] = 0.f;
    if (c < len) {                              // VEC > 1: dim, vdim and rot / 2 are multiples of VEC
      load_vec<VEC>(src + c, f);
      if (w != nullptr) {
        float g[VEC];
        load_vec<VEC>(w + c, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) f[i] = f[i] * r * g[i];
        if (c < p.rot) {
          const bool low = c < half;
          const int oc = low ? c + half : c - half, a = low ? c : oc;
          float o[VEC], cs[VEC], sn[VEC];
          load_vec<VEC>(src + oc, o);
          load_vec<VEC>(w + oc, g);
          load_vec<VEC>(p.cos_sin + (long long)pos * half + a, cs);
          load_vec<VEC>(p.cos_sin + ((long long)p.ctx + pos) * half + a, sn);
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            const float other = o[i] * r * g[i];
            f[i] = low ? f[i] * cs[i] - other * sn[i] : f[i] * cs[i] + other * sn[i];
          }
        }
      }
    }
    store_vec<VEC>(dst + c, f);
  }
}

// The same for sizes in whole pieces of 8 elements: LPV lanes own a vector, one piece each; a thread owns the same columns of UNITS
// vectors of one row, so it loads the angles once.
template <typename T, int LPV, int UNITS>
__global__ void __launch_bounds__(512, 2) grouped_prep_pieces_kernel(const GroupedPrepParams p) {
  pdl_sync();
  const int row = blockIdx.x, piece = threadIdx.x % LPV, c = piece * 8;
  const int nq = p.heads * p.maps, nk = p.wk != nullptr ? p.kv_heads * p.maps : 0, nv = p.wk != nullptr ? p.kv_heads : 0;
  const int per = blockDim.x / LPV, v0 = blockIdx.y * per * UNITS + threadIdx.x / LPV;       // vectors v0, v0 + per, ...
  const T* src = reinterpret_cast<const T*>(p.proj) + (long long)row * p.ld;
  const int half = p.rot / 2, shift = half / 8;
  const bool low = c < half, turned = c < p.rot;
  const int partner = turned ? (low ? piece + shift : piece - shift) : piece;    // lane that holds the other half of the pairs
  const uint32_t lanes = LPV == 32 ? 0xffffffffu : (((1u << (LPV & 31)) - 1u) << ((threadIdx.x & 31) / LPV * LPV));
  auto offset = [&](int v) { return v >= nq + nk ? (nq + nk) * p.dim + (v - nq - nk) * p.vdim : v * p.dim; };    // q | k | v
  Piece<T> raw[UNITS];
#pragma unroll
  for (int u = 0; u < UNITS; ++u) {                              // everything is requested before the first vector is worked on
    const int v = v0 + u * per;
#pragma unroll
    for (int j = 0; j < (int)sizeof(T) / 2; ++j) raw[u].v[j] = make_uint4(0, 0, 0, 0);
    if (v < nq + nk + nv && c < (v >= nq + nk ? p.vdim : p.dim)) raw[u] = load_piece(src + offset(v) + c);
  }
  float cs[8], sn[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) cs[j] = sn[j] = 0.f;
  if (turned) {
    int at = p.positions[row];
    if (at < 0 || at >= p.ctx) {
      if (threadIdx.x == 0) report_bad_arg(p.status, 14);
      at = 0;
    }
    const float* tab = p.cos_sin + (long long)at * half + (low ? c : c - half);
    unpack(load_piece(tab), cs);
    unpack(load_piece(tab + (long long)p.ctx * half), sn);
    if (low) {
#pragma unroll
      for (int j = 0; j < 8; ++j) sn[j] = -sn[j];
    }
  }
  const long long slot = p.slots[row];
  const bool keep = slot >= 0 && slot < p.num_slots;             // a padding row of the batch has no slot
  if (nk > 0 && slot >= p.num_slots && threadIdx.x == 0) report_bad_arg(p.status, 13);
  T* cache = reinterpret_cast<T*>(p.cache) + (keep ? slot : 0) * ((long long)p.kv_heads * (p.maps * p.kp + p.vp));
#pragma unroll
  for (int u = 0; u < UNITS; ++u) {
    const int v = v0 + u * per;
    if (v >= nq + nk + nv) break;
    const bool query = v < nq, value = v >= nq + nk;
    float f[8];
    unpack(raw[u], f);
    if (!value) {
      float w[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) w[j] = 0.f;
      if (c < p.dim) unpack(load_piece(reinterpret_cast<const T*>(query ? p.wq : p.wk) + c), w);
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
#pragma unroll
      for (int o = LPV / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(lanes, ss, o);
      const float r = rsqrtf(ss / (float)p.dim + p.eps);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= r * w[j];
      if (p.rot > 0) {
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const float o = __shfl_sync(lanes, f[j], partner, LPV);
          if (turned) f[j] = fmaf(f[j], cs[j], o * sn[j]);
        }
      }
    }
    if (query) {
      if (c < p.qp) store8(reinterpret_cast<T*>(p.q) + ((long long)row * nq + v) * p.qp + c, f);    // lanes past dim: zeros, the pad
      continue;
    }
    if (!keep) continue;
    T* dst = cache + (value ? nk * p.kp + (v - nq - nk) * p.vp : (v - nq) * p.kp);
    if (c < (value ? p.vdim : p.dim)) store8(dst + c, f);
    if (value)
      for (int e = c + LPV * 8; e < p.vdim; e += LPV * 8) {      // values longer than a key: copied
        float g[8];
        unpack(load_piece(src + offset(v) + e), g);
        store8(dst + e, g);
      }
  }
}

template <typename T, int LPV>
static void launch_prep_lanes(const GroupedPrepParams& p, int vectors, cudaStream_t st) {
  const bool many = p.rows >= 148 * 16;                          // few rows: their vectors spread over the SMs
  const int units = many ? 4 : 1;
  int threads = ((vectors + units - 1) / units * LPV + 31) / 32 * 32;
  if (threads > 512) threads = 256;
  const int per = threads / LPV * units;
  const dim3 grid(p.rows, (unsigned)((vectors + per - 1) / per));
  if (many) launch_dep(grouped_prep_pieces_kernel<T, LPV, 4>, grid, threads, 0, st, p);
  else launch_dep(grouped_prep_pieces_kernel<T, LPV, 1>, grid, threads, 0, st, p);
}

template <typename T>
static void launch_prep_pieces(const GroupedPrepParams& p, cudaStream_t st) {
  const int vectors = p.heads * p.maps + (p.wk != nullptr ? p.kv_heads * (p.maps + 1) : 0);
  if (p.dim <= 64) launch_prep_lanes<T, 8>(p, vectors, st);
  else if (p.dim <= 128) launch_prep_lanes<T, 16>(p, vectors, st);
  else launch_prep_lanes<T, 32>(p, vectors, st);
}

// Norm over the whole projection: the queries of all heads share one root mean square, so do the keys; weights of the projections'
// sizes.  One block per row, pieces of VEC elements per thread, the first KEEP of them in registers between the passes.
template <typename T, int VEC>
__global__ void __launch_bounds__(512, 2) grouped_prep_whole_kernel(const GroupedPrepParams p) {
  pdl_sync();
  __shared__ float red[2][16];
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool own = p.wk != nullptr;
  const int nq = p.heads * p.dim, nk = own ? p.kv_heads * p.dim : 0, nv = own ? p.kv_heads * p.vdim : 0;
  const T* src = reinterpret_cast<const T*>(p.proj) + (long long)row * p.ld;
  const int step = blockDim.x * VEC, total = nq + nk + nv;
  auto load = [&](const T* from, float (&f)[VEC]) __attribute__((always_inline)) {
    if constexpr (VEC == 8) unpack(load_piece(from), f);
    else f[0] = to_f(*from);
  };
  constexpr int KEEP = 2;
  float keep[KEEP][VEC], sq = 0.f, sk = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x * VEC + j * step;
#pragma unroll
    for (int i = 0; i < VEC; ++i) keep[j][i] = 0.f;
    if (c < total) load(src + c, keep[j]);
  }
  int pos = p.positions[row];
  const long long slot = p.slots[row];
  auto square = [&](int c, const float (&f)[VEC]) __attribute__((always_inline)) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(f[i], f[i], ss);
    if (c < nq) sq += ss;
    else if (c < nq + nk) sk += ss;
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j) square(threadIdx.x * VEC + j * step, keep[j]);
  for (int c = threadIdx.x * VEC + KEEP * step; c < nq + nk; c += step) {
    float f[VEC];
    load(src + c, f);
    square(c, f);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    sk += __shfl_xor_sync(0xffffffffu, sk, o);
  }
  if (lane == 0) {
    red[0][warp] = sq;
    red[1][warp] = sk;
  }
  __syncthreads();
  sq = sk = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) {
    sq += red[0][w];
    sk += red[1][w];
  }
  const float rq = rsqrtf(sq / (float)nq + p.eps), rk = own ? rsqrtf(sk / (float)nk + p.eps) : 0.f;
  if (p.rot > 0 && (pos < 0 || pos >= p.ctx)) {
    if (threadIdx.x == 0) report_bad_arg(p.status, 23);
    pos = 0;
  }
  const bool live = slot >= 0 && slot < p.num_slots;             // a padding row of the batch has no slot
  if (own && slot >= p.num_slots && threadIdx.x == 0) report_bad_arg(p.status, 24);
  T* cache = reinterpret_cast<T*>(p.cache) + (live ? slot : 0) * ((long long)p.kv_heads * (p.kp + p.vp));
  T* q = reinterpret_cast<T*>(p.q) + (long long)row * p.heads * p.qp;
  const int half = p.rot / 2;
  auto finish = [&](int c, float (&f)[VEC]) __attribute__((always_inline)) {
    const bool query = c < nq, vector = c < nq + nk;
    const int at = query ? c : c - nq, v = vector ? at / p.dim : 0, e = at - v * p.dim;
    const T* w = reinterpret_cast<const T*>(query ? p.wq : p.wk) + at;
    const float r = query ? rq : rk;
    const bool turned = vector && e < p.rot, low = e < half;
    if (vector) {
      float g[VEC];
      load(w, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) f[i] *= r * g[i];
    }
    if (p.rot > 0) {
      const int to = low ? half : -half;
      float o[VEC];
      if (turned) {                          // the other half of the pair, normed again
        float g[VEC];
        load(src + c + to, o);
        load(w + to, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) o[i] *= r * g[i];
      }
      if (turned) {
        const float* cp = p.cos_sin + (long long)pos * half + (low ? e : e - half);
        const float* sp = cp + (long long)p.ctx * half;
        float cs[VEC], sn[VEC];
        if constexpr (VEC == 8) {
          unpack(load_piece(cp), cs);
          unpack(load_piece(sp), sn);
        } else {
          cs[0] = *cp;
          sn[0] = *sp;
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) f[i] = low ? f[i] * cs[i] - o[i] * sn[i] : f[i] * cs[i] + o[i] * sn[i];
      }
    }
    if (!query && !live) return;
    T* dst;
    if (query) {
      dst = q + v * p.qp + e;
    } else if (vector) {
      dst = cache + v * p.kp + e;
    } else {
      const int a = c - nq - nk, n = a / p.vdim;
      dst = cache + p.kv_heads * p.kp + n * p.vp + (a - n * p.vdim);
    }
    if constexpr (VEC == 8) store8(dst, f);
    else from_f(*dst, f[0]);
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x * VEC + j * step;
    if (c < total) finish(c, keep[j]);
  }
  for (int c = threadIdx.x * VEC + KEEP * step; c < total; c += step) {
    float f[VEC];
    load(src + c, f);
    finish(c, f);
  }
  // the pads behind every vector
  auto pad = [&](T* base, int vectors, int pitch, int len) {
    const int n = pitch - len;
    for (int i = threadIdx.x; i < vectors * n; i += blockDim.x) from_f(base[(i / n) * pitch + len + i % n], 0.f);
  };
  if (p.qp > p.dim) pad(q, p.heads, p.qp, p.dim);
  if (own && live && p.kp > p.dim) pad(cache, p.kv_heads, p.kp, p.dim);
  if (own && live && p.vp > p.vdim) pad(cache + p.kv_heads * p.kp, p.kv_heads, p.vp, p.vdim);
}

// The same where a thread's pieces of 8 elements have the same place in their vectors (dim a power of two up to 256): weights and angles are
// requested with the pieces, before the block waits for its sums, the angles once, and the other half of a rotated pair comes
// from the lane that holds it.
template <typename T>
__global__ void __launch_bounds__(512, 2) grouped_prep_whole_pieces_kernel(const GroupedPrepParams p) {
  pdl_sync();
  __shared__ float red[2][16];
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool own = p.wk != nullptr;
  const int nq = p.heads * p.dim, nk = own ? p.kv_heads * p.dim : 0, total = nq + nk + (own ? p.kv_heads * p.vdim : 0);
  const T* src = reinterpret_cast<const T*>(p.proj) + (long long)row * p.ld;
  const int step = blockDim.x * 8, c0 = threadIdx.x * 8, e = c0 & (p.dim - 1);      // e: place in the vector
  const int half = p.rot / 2;
  const bool turned = e < p.rot, low = e < half;
  const int from = turned ? lane + (low ? half : -half) / 8 : lane;
  auto weights = [&](int c) { return c < nq ? reinterpret_cast<const T*>(p.wq) + c : reinterpret_cast<const T*>(p.wk) + (c - nq); };
  constexpr int KEEP = 2;
  Piece<T> raw[KEEP], w[KEEP];
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
#pragma unroll
    for (int i = 0; i < (int)sizeof(T) / 2; ++i) raw[j].v[i] = w[j].v[i] = make_uint4(0, 0, 0, 0);
    if (c0 + j * step < total) raw[j] = load_piece(src + c0 + j * step);
  }
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if (c0 + j * step < nq + nk) w[j] = load_piece(weights(c0 + j * step));
  int pos = p.positions[row];
  const long long slot = p.slots[row];
  if (p.rot > 0 && (pos < 0 || pos >= p.ctx)) {
    if (threadIdx.x == 0) report_bad_arg(p.status, 23);
    pos = 0;
  }
  float cs[8], sn[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) cs[i] = sn[i] = 0.f;
  if (turned) {
    const float* cp = p.cos_sin + (long long)pos * half + (low ? e : e - half);
    unpack(load_piece(cp), cs);
    unpack(load_piece(cp + (long long)p.ctx * half), sn);
    if (low) {
#pragma unroll
      for (int i = 0; i < 8; ++i) sn[i] = -sn[i];
    }
  }
  float sq = 0.f, sk = 0.f;
  auto square = [&](int c, const Piece<T>& r) __attribute__((always_inline)) {
    float f[8], ss = 0.f;
    unpack(r, f);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(f[i], f[i], ss);
    if (c < nq) sq += ss;
    else if (c < nq + nk) sk += ss;
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j) square(c0 + j * step, raw[j]);
  for (int c = c0 + KEEP * step; c < nq + nk; c += step) square(c, load_piece(src + c));
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    sk += __shfl_xor_sync(0xffffffffu, sk, o);
  }
  if (lane == 0) {
    red[0][warp] = sq;
    red[1][warp] = sk;
  }
  __syncthreads();
  sq = lane < (int)(blockDim.x >> 5) ? red[0][lane & 15] : 0.f;
  sk = lane < (int)(blockDim.x >> 5) ? red[1][lane & 15] : 0.f;
#pragma unroll
  for (int o = 8; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    sk += __shfl_xor_sync(0xffffffffu, sk, o);
  }
  sq = __shfl_sync(0xffffffffu, sq, 0);
  sk = __shfl_sync(0xffffffffu, sk, 0);
  const float rq = rsqrtf(sq / (float)nq + p.eps), rk = own ? rsqrtf(sk / (float)nk + p.eps) : 0.f;
  const bool live = slot >= 0 && slot < p.num_slots;             // a padding row of the batch has no slot
  if (own && slot >= p.num_slots && threadIdx.x == 0) report_bad_arg(p.status, 24);
  T* cache = reinterpret_cast<T*>(p.cache) + (live ? slot : 0) * ((long long)p.kv_heads * (p.kp + p.vp));
  T* q = reinterpret_cast<T*>(p.q) + (long long)row * p.heads * p.qp;
  auto finish = [&](int c, const Piece<T>& r, const Piece<T>& wr) __attribute__((always_inline)) {      // all lanes of a warp together
    const bool query = c < nq, vector = c < nq + nk;
    const int at = query ? c : c - nq, v = vector ? at / p.dim : 0;
    float f[8];
    unpack(r, f);
    if (vector) {
      float g[8];
      unpack(wr, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] *= (query ? rq : rk) * g[i];
    }
    if (p.rot > 0) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float o = __shfl_sync(0xffffffffu, f[i], from);
        if (turned && vector) f[i] = fmaf(f[i], cs[i], o * sn[i]);
      }
    }
    if (c >= total || (!query && !live)) return;
    if (query) {
      store8(q + v * p.qp + e, f);
    } else if (vector) {
      store8(cache + v * p.kp + e, f);
    } else {
      const int a = c - nq - nk, n = a / p.vdim;
      store8(cache + p.kv_heads * p.kp + n * p.vp + (a - n * p.vdim), f);
    }
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if (__any_sync(0xffffffffu, c0 + j * step < total)) finish(c0 + j * step, raw[j], w[j]);
  for (int k = KEEP * step; k < total; k += step) {
    const int c = c0 + k;
    Piece<T> r, wr;
#pragma unroll
    for (int i = 0; i < (int)sizeof(T) / 2; ++i) r.v[i] = wr.v[i] = make_uint4(0, 0, 0, 0);
    if (c < total) r = load_piece(src + c);
    if (c < nq + nk) wr = load_piece(weights(c));
    finish(c, r, wr);
  }
  if (p.qp > p.dim)                          // a query's pitch is 64 at least
    for (int i = threadIdx.x; i < p.heads * (p.qp - p.dim); i += blockDim.x)
      from_f(q[(i / (p.qp - p.dim)) * p.qp + p.dim + i % (p.qp - p.dim)], 0.f);
}

// ------------------------------------------------------------------------------------------------------ general form
// One warp per (row, head), keys one after the other; any size, T = bf16 or fp32.  row_seq[row] names the row's line of
// `tables` (null: line `row`).
struct GroupedRowsParams {
  const void *q, *cache, *gate;
  void* o;
  long long ld_o, ld_gate;
  const float* bias;
  const int *row_seq, *positions, *tables;
  const long long* slots;
  int bias_len, seqs, rows, max_pages, page_size, num_pages;
  GroupedShape s;
  uint32_t* status;
};

template <typename T>
__global__ void __launch_bounds__(128) grouped_rows_kernel(const GroupedRowsParams p) {
  pdl_sync();
  extern __shared__ float gsm[];
  const GroupedShape& s = p.s;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + warp;
  if (item >= (long long)p.rows * s.heads) return;
  const int row = (int)(item / s.heads), h = (int)(item - (long long)row * s.heads);
  float* qs = gsm + warp * s.maps * (s.dim + s.vdim);
  float* acc = qs + s.maps * s.dim;
  const T* qr = reinterpret_cast<const T*>(p.q) + ((long long)row * s.heads + h) * s.maps * s.qp;
  for (int m = 0; m < s.maps; ++m) {
    for (int c = lane; c < s.dim; c += 32) qs[m * s.dim + c] = to_f(qr[m * s.qp + c]);
    for (int c = lane; c < s.vdim; c += 32) acc[m * s.vdim + c] = 0.f;
  }
  __syncwarp();
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const int seq = p.row_seq != nullptr ? p.row_seq[row] : row;
  const bool live = p.slots[row] >= 0 && seq >= 0 && seq < p.seqs;
  const int pos = p.positions[row], g = h / (s.heads / s.kv_heads);
  const int width = s.kv_heads * (s.maps * s.kp + s.vp);
  if (live) {
    const int* table = p.tables + (long long)seq * p.max_pages;
    const int lo = max(0, first_seen(s, pos)), kept = min(s.keep, lo);
    const float slope = s.slopes != nullptr ? s.slopes[h] : 0.f;
    for (int n = lo - kept; n <= pos; ++n) {
      const int j = n < lo ? n - (lo - kept) : n;                 // the kept positions, then the window
      const int pg = j / p.page_size;
      const int page = pg < p.max_pages ? table[pg] : -1;
      if ((unsigned)page >= (unsigned)p.num_pages) {
        if (lane == 0) report_bad_arg(p.status, 15);
        break;
      }
      const T* c = reinterpret_cast<const T*>(p.cache) + ((long long)page * p.page_size + j % p.page_size) * width;
      const T* v = c + s.kv_heads * s.maps * s.kp + g * s.vp;
      const float b = (p.bias != nullptr ? p.bias[h * p.bias_len + min(pos - j, p.bias_len - 1)] : 0.f) - slope * (float)(pos - j);
      for (int m = 0; m < s.maps; ++m) {
        const T* k = c + (g * s.maps + m) * s.kp;
        float sc = 0.f;
        for (int i = lane; i < s.dim; i += 32) sc = fmaf(qs[m * s.dim + i], to_f(k[i]), sc);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) sc += __shfl_xor_sync(0xffffffffu, sc, o);
        sc *= s.scale;
        if (s.softcap > 0.f) sc = s.softcap * tanhf(sc / s.softcap);
        sc += b;
        const float mn = fmaxf(mx[m], sc);
        const float a = expf(mx[m] - mn), e = expf(sc - mn);      // first key: exp(-inf) = 0
        l[m] = l[m] * a + e;
        for (int i = lane; i < s.vdim; i += 32) acc[m * s.vdim + i] = acc[m * s.vdim + i] * a + e * to_f(v[i]);
        mx[m] = mn;
      }
    }
  }
  if (s.sink != nullptr && live) {
    const float mn = fmaxf(mx[0], s.sink[h]);
    const float a = expf(mx[0] - mn);
    l[0] = l[0] * a + expf(s.sink[h] - mn);
    for (int c = lane; c < s.vdim; c += 32) acc[c] *= a;
  }
  const float i0 = l[0] > 0.f ? 1.f / l[0] : 0.f, i1 = l[1] > 0.f ? s.difference / l[1] : 0.f;
  float ss = 0.f;
  for (int c = lane; c < s.vdim; c += 32) {
    float o = acc[c] * i0;
    if (s.maps == 2) o -= acc[s.vdim + c] * i1;
    acc[c] = o;
    ss = fmaf(o, o, ss);
  }
  float f = 1.f;
  if (s.maps == 2) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    f = rsqrtf(ss / (float)s.vdim + s.eps) * s.out_scale;
  }
  T* orow = reinterpret_cast<T*>(p.o) + (long long)row * p.ld_o + h * s.vdim;
  const T* grow = p.gate != nullptr ? reinterpret_cast<const T*>(p.gate) + (long long)row * p.ld_gate + gate_column(s, h) : nullptr;
  for (int c = lane; c < s.vdim; c += 32) {
    float o = acc[c] * f;
    if (grow != nullptr) o /= 1.f + expf(-to_f(grow[s.head_gate ? 0 : c]));
    from_f(orow[c], live ? o : 0.f);
  }
}

// ----------------------------------------------------------------------------------------------- decode, bf16, mma.sync
// One CTA = one request, up to 16 query vectors (heads x maps) of one key/value head, one split of the window.  The vectors
// are the M = 16 rows of mma.sync, so a cached byte is read once for all of them; with two maps a query vector is zero
// outside its own map's columns and both maps' keys are one key of twice the length.
// The four warps work on their own tiles of 16 tokens (round robin): own ring (bulk copies, one per token and key or value, a lane
// each), own softmax state (online, in fragments), own output; nothing is shared before the end, so the loop has no block
// barrier.
constexpr int GD_WARPS = 4, GD_STAGES = 3, GD_TOK = 16;

__device__ __forceinline__ void gd_ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void gd_ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void gd_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
struct GroupedDecodeParams {
  const __nv_bfloat16 *q, *cache, *gate;
  __nv_bfloat16* o;
  long long ld_o, ld_gate;
  float *part_o, *part_ml;        // splits > 1: (rows, heads, maps, splits, vdim) and (..., 2)
  const float* bias;
  const int *positions, *tables;
  const long long* slots;
  int bias_len, rows, max_pages, page_size, num_pages, splits, groups;     // groups of 16 query vectors per key/value head
  GroupedShape s;
  uint32_t* status;
};

template <int KT, int VT>         // 16-column steps of a key (both maps), 8-column tiles of a value
struct GroupedDecodeSmem {
  static constexpr int KPITCH = KT * 16 + 8, VPITCH = VT * 8 + 8;          // odd numbers of 16-byte pieces
  static constexpr int STAGE = GD_TOK * (KPITCH + VPITCH);                 // elements
  static constexpr int RING = GD_WARPS * GD_STAGES * STAGE * 2;
  static constexpr int OPITCH = VT * 8 + 4;
  static constexpr int MERGE = GD_WARPS * (16 * OPITCH + 32) * 4;
  static constexpr int OFF_BAR = RING > MERGE ? RING : MERGE;              // a barrier per warp and stage, the abort word
  static constexpr int TOTAL = OFF_BAR + GD_WARPS * GD_STAGES * 8 + 16;
};

// Heads of one row from their merged maps: value(m, c) gives map m's normalised output.  One warp per head.
template <typename F>
__device__ __forceinline__ void grouped_finish(const GroupedShape& s, int lane, __nv_bfloat16* orow, const __nv_bfloat16* grow, F value) {
  float o[8], ss = 0.f;            // vdim <= 256
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int c = lane + i * 32;
    o[i] = 0.f;
    if (c < s.vdim) {
      o[i] = value(0, c);
      if (s.maps == 2) o[i] -= s.difference * value(1, c);
    }
    ss = fmaf(o[i], o[i], ss);
  }
  float f = 1.f;
  if (s.maps == 2) {
#pragma unroll
    for (int k = 16; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
    f = rsqrtf(ss / (float)s.vdim + s.eps) * s.out_scale;
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int c = lane + i * 32;
    if (c >= s.vdim) break;
    float x = o[i] * f;
    if (grow != nullptr) x *= sigmoid_f(__bfloat162float(grow[s.head_gate ? 0 : c]));
    orow[c] = __float2bfloat16(x);
  }
}

// Denominator l relative to the maximum m (log2 units; -inf: no key), with the sink in it.
__device__ __forceinline__ void add_sink(float sink, float m, float& l) {
  if (m != -INFINITY) l += exp2f(fminf(fmaf(sink, LOG2E, -m), 126.f));      // a sink that far above every key takes all the weight
}

template <int KT, int VT>
__global__ void __launch_bounds__(GD_WARPS * 32) grouped_decode_kernel(const GroupedDecodeParams p) {
  using L = GroupedDecodeSmem<KT, VT>;
  extern __shared__ __align__(16) uint8_t gd_smem[];
  const GroupedShape& s = p.s;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // the key/value heads of a row are neighbours: they read neighbouring parts of the same cache rows at about the same time
  const int g = blockIdx.x / p.groups, grp = blockIdx.x - g * p.groups, row = blockIdx.y, split = blockIdx.z;
  const int per_kv = s.heads / s.kv_heads, hpg = 16 / s.maps;              // query heads per key/value head and per CTA
  const int h0 = g * per_kv + grp * hpg, nh = min(hpg, per_kv - grp * hpg);
  const int kd = s.maps * s.kp;
  const int width = s.kv_heads * (kd + s.vp);
  __nv_bfloat16* ring = reinterpret_cast<__nv_bfloat16*>(gd_smem) + warp * GD_STAGES * L::STAGE;
  uint64_t* full = reinterpret_cast<uint64_t*>(gd_smem + L::OFF_BAR) + warp * GD_STAGES;
  volatile uint32_t* abort_word = reinterpret_cast<uint32_t*>(gd_smem + L::OFF_BAR + GD_WARPS * GD_STAGES * 8);
  // pad columns, and the places of tokens that are not seen, stay finite
  for (int i = lane; i < GD_STAGES * L::STAGE / 8; i += 32) reinterpret_cast<uint4*>(ring)[i] = make_uint4(0, 0, 0, 0);
  if (lane == 0) {
    for (int i = 0; i < GD_STAGES; ++i) mbar_init(&full[i], 1);
    fence_barrier_init();
  }
  if (threadIdx.x == 0) *abort_word = 0;
  fence_proxy_async_smem();
  __syncthreads();
  pdl_sync();
  const int pos = p.positions[row];
  const bool live = p.slots[row] >= 0 && pos >= 0;
  const int lo = live ? max(0, first_seen(s, pos)) : 0;
  // tiles of 16 tokens, starting at multiples of 16: those of the kept tokens in front of the window's first tile, then the window's
  const int first = lo / GD_TOK, kept = min((s.keep + GD_TOK - 1) / GD_TOK, first);
  const int total = live ? kept + pos / GD_TOK + 1 - first : 0;
  auto token = [&](int tile) { return (tile < kept ? tile : first + tile - kept) * GD_TOK; };
  const int per = (total + p.splits - 1) / p.splits;
  const int i0 = min(total, split * per), tiles = min(total, i0 + per) - i0;
  const int* table = p.tables + (long long)row * p.max_pages;

  auto look_up = [&](int i) -> long long {     // cache row of this lane's token of tile i0 + i of this split; -1: none
    if (i >= tiles) return -1;
    const int t = token(i0 + i) + (lane & 15);
    if ((t < lo && t >= s.keep) || t > pos) return -1;
    const int pg = t / p.page_size;
    const int page = pg < p.max_pages ? table[pg] : -1;
    if ((unsigned)page < (unsigned)p.num_pages) return (long long)page * p.page_size + t % p.page_size;
    report_bad_arg(p.status, 16);
    return -1;
  };
  const uint32_t k_bytes = (uint32_t)kd * 2, v_bytes = (uint32_t)s.vp * 2;
  const int from = lane < 16 ? g * kd : s.kv_heads * kd + g * s.vp;            // lanes 0 - 15: keys, 16 - 31: values
  auto request = [&](int i, long long src) {
    const int st = (i / GD_WARPS) % GD_STAGES;
    __nv_bfloat16* k = ring + st * L::STAGE;
    const uint32_t seen = __ballot_sync(0xffffffffu, src >= 0) & 0xffffu;
    if (lane == 0) mbar_expect_tx(&full[st], __popc(seen) * (k_bytes + v_bytes));
    __syncwarp();
    if (src >= 0)
      bulk_load(lane < 16 ? k + lane * L::KPITCH : k + GD_TOK * L::KPITCH + (lane - 16) * L::VPITCH, p.cache + src * width + from,
                lane < 16 ? k_bytes : v_bytes, &full[st]);
  };
#pragma unroll
  for (int n = 0; n < GD_STAGES; ++n)
    if (warp + n * GD_WARPS < tiles) request(warp + n * GD_WARPS, look_up(warp + n * GD_WARPS));
  long long next = look_up(warp + GD_STAGES * GD_WARPS);            // looked up a tile earlier than it is requested
  // query fragments: vector r = head * maps + map, columns of its own map only
  uint32_t qf[KT][4];
#pragma unroll
  for (int k = 0; k < KT; ++k)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (lane >> 2) + (i & 1) * 8, col = k * 16 + (i >> 1) * 8 + (lane & 3) * 2;
      const int hl = r / s.maps, m = r - hl * s.maps, c = col - m * s.kp;
      qf[k][i] = 0;
      if (hl < nh && c >= 0 && c < s.kp)
        qf[k][i] = *reinterpret_cast<const uint32_t*>(p.q + (((long long)row * s.heads + h0 + hl) * s.maps + m) * s.qp + c);
    }
  float acc[VT][4], mrun[2] = {-INFINITY, -INFINITY}, lrun[2] = {0.f, 0.f};
#pragma unroll
  for (int j = 0; j < VT; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
  const float scale_log2 = s.scale * LOG2E, slope = s.softcap > 0.f ? 2.f * LOG2E * s.scale / s.softcap : 0.f;
  const float* bias[2] = {nullptr, nullptr};
  if (p.bias != nullptr) {
#pragma unroll
    for (int i = 0; i < 2; ++i) bias[i] = p.bias + (long long)(h0 + min(((lane >> 2) + i * 8) / s.maps, nh - 1)) * p.bias_len;
  }

  float slope2[2] = {0.f, 0.f};                        // log2 units per token, of this lane's two query vectors
  if (s.slopes != nullptr) {
#pragma unroll
    for (int i = 0; i < 2; ++i) slope2[i] = LOG2E * s.slopes[h0 + min((lane >> 2) + i * 8, nh - 1)];
  }
  float bn[2][4];                                      // bias of the tile after the one at work
  auto load_bias = [&](int i) {
    const int t = token(i0 + i) + (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) bn[n][e] = __ldg(bias[e >> 1] + max(0, min(pos - (t + n * 8 + (e & 1)), p.bias_len - 1)));
  };
  if (p.bias != nullptr) load_bias(warp);

  for (int i = warp; i < tiles; i += GD_WARPS) {
    const int round = i / GD_WARPS, st = round % GD_STAGES;
    const bool landed = mbar_wait(&full[st], (round / GD_STAGES) & 1, abort_word);
    if (!__all_sync(0xffffffffu, landed)) {
      *abort_word = ERR_WAIT_FULL;
      break;
    }
    const __nv_bfloat16* k = ring + st * L::STAGE;
    const __nv_bfloat16* v = k + GD_TOK * L::KPITCH;
    float sc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    const uint32_t k_addr = smem_u32(k + ((lane & 7) + (lane >> 4) * 8) * L::KPITCH + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int kk = 0; kk < KT; ++kk) {
      uint32_t b[4];
      gd_ldsm_x4(b, k_addr + kk * 32);
      gd_mma(sc[0], qf[kk], b[0], b[1]);
      gd_mma(sc[1], qf[kk], b[2], b[3]);
    }
    const int t0 = token(i0 + i) + (lane & 3) * 2;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = t0 + n * 8 + (e & 1);
        float x = s.softcap > 0.f ? capped_log2(sc[n][e], slope, s.softcap * LOG2E) : sc[n][e] * scale_log2;
        const bool seen = (t >= lo || t < s.keep) && t <= pos;
        if (p.bias != nullptr) x = fmaf(bn[n][e], LOG2E, x);
        else x = fmaf(slope2[e >> 1], (float)(t - pos), x);
        x = seen ? x : -INFINITY;
        sc[n][e] = x;
        mx[e >> 1] = fmaxf(mx[e >> 1], x);
      }
    if (p.bias != nullptr && i + GD_WARPS < tiles) load_bias(i + GD_WARPS);
    float alpha[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      const float mn = fmaxf(mrun[r], mx[r]);          // finite: every tile holds a token that is seen
      alpha[r] = exp2f(mrun[r] - mn);
      mrun[r] = mn;
      lrun[r] *= alpha[r];
    }
    uint32_t pf[4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float a = exp2f(sc[n][r * 2] - mrun[r]), b = exp2f(sc[n][r * 2 + 1] - mrun[r]);
        lrun[r] += a + b;
        pf[n * 2 + r] = pack_bf16x2(a, b);
      }
    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
      for (int j = 0; j < VT; ++j) {
        acc[j][0] *= alpha[0]; acc[j][1] *= alpha[0]; acc[j][2] *= alpha[1]; acc[j][3] *= alpha[1];
      }
    }
    const uint32_t v_addr = smem_u32(v + ((lane & 7) + ((lane >> 3) & 1) * 8) * L::VPITCH + (lane >> 4) * 8);
#pragma unroll
    for (int j = 0; j < VT / 2; ++j) {
      uint32_t b[4];
      gd_ldsm_x4_t(b, v_addr + j * 32);
      gd_mma(acc[2 * j], pf, b[0], b[1]);
      gd_mma(acc[2 * j + 1], pf, b[2], b[3]);
    }
    __syncwarp();                                      // everybody has read the stage
    if (i + GD_STAGES * GD_WARPS < tiles) {
      request(i + GD_STAGES * GD_WARPS, next);
      next = look_up(i + (GD_STAGES + 1) * GD_WARPS);
    }
  }
  __syncthreads();                                     // the rings become the merge buffer
  if (*abort_word != 0) {                              // give copies that may still be in flight time to land
    if (threadIdx.x == 0 && p.status != nullptr) atomicCAS(p.status, 0u, *abort_word | (blockIdx.x << 8));
    const uint64_t w0 = globaltimer_ns();
    while (globaltimer_ns() - w0 < 200000ull) __nanosleep(1000);
  }
  __syncthreads();
  float* mo = reinterpret_cast<float*>(gd_smem) + warp * (16 * L::OPITCH + 32);
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    lrun[r] += __shfl_xor_sync(0xffffffffu, lrun[r], 1);
    lrun[r] += __shfl_xor_sync(0xffffffffu, lrun[r], 2);
    const int vr = (lane >> 2) + r * 8;
    if ((lane & 3) == 0) {
      mo[16 * L::OPITCH + vr] = mrun[r];
      mo[16 * L::OPITCH + 16 + vr] = lrun[r];
    }
#pragma unroll
    for (int j = 0; j < VT; ++j)
      *reinterpret_cast<float2*>(mo + vr * L::OPITCH + j * 8 + (lane & 3) * 2) = make_float2(acc[j][r * 2], acc[j][r * 2 + 1]);
  }
  __syncthreads();
  const float* mb = reinterpret_cast<const float*>(gd_smem);
  for (int hl = warp; hl < nh; hl += GD_WARPS) {
    float f[2][GD_WARPS], m[2], l[2];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
      m[mp] = -INFINITY;
      l[mp] = 0.f;
      if (mp >= s.maps) continue;
      const int r = hl * s.maps + mp;
#pragma unroll
      for (int w = 0; w < GD_WARPS; ++w) m[mp] = fmaxf(m[mp], mb[w * (16 * L::OPITCH + 32) + 16 * L::OPITCH + r]);
#pragma unroll
      for (int w = 0; w < GD_WARPS; ++w) {
        const float* ml = mb + w * (16 * L::OPITCH + 32) + 16 * L::OPITCH;
        f[mp][w] = ml[r] == -INFINITY ? 0.f : exp2f(ml[r] - m[mp]);
        l[mp] += ml[16 + r] * f[mp][w];
      }
    }
    auto sum = [&](int mp, int c) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < GD_WARPS; ++w) v += f[mp][w] * mb[w * (16 * L::OPITCH + 32) + (hl * s.maps + mp) * L::OPITCH + c];
      return v;
    };
    const int h = h0 + hl;
    if (p.splits > 1) {
#pragma unroll
      for (int mp = 0; mp < 2; ++mp) {
        if (mp >= s.maps) break;
        const long long at = (((long long)row * s.heads + h) * s.maps + mp) * p.splits + split;
        if (lane == 0) {
          p.part_ml[at * 2] = m[mp];
          p.part_ml[at * 2 + 1] = l[mp];
        }
        for (int c = lane; c < s.vdim; c += 32) p.part_o[at * s.vdim + c] = sum(mp, c);
      }
    } else {
      if (s.sink != nullptr) add_sink(s.sink[h], m[0], l[0]);
      const float inv[2] = {l[0] > 0.f ? 1.f / l[0] : 0.f, l[1] > 0.f ? 1.f / l[1] : 0.f};
      grouped_finish(s, lane, p.o + (long long)row * p.ld_o + h * s.vdim,
                     p.gate != nullptr ? p.gate + (long long)row * p.ld_gate + gate_column(s, h) : nullptr, [&](int mp, int c) {
                       float v = 0.f;                  // constant map index: the factors stay in registers
#pragma unroll
                       for (int w = 0; w < GD_WARPS; ++w)
                         v += (mp ? f[1][w] : f[0][w]) * mb[w * (16 * L::OPITCH + 32) + (hl * s.maps + mp) * L::OPITCH + c];
                       return v * (mp ? inv[1] : inv[0]);
                     });
    }
  }
}

// Splits of one row: one warp per (row, head).
__global__ void __launch_bounds__(128) grouped_merge_kernel(const GroupedDecodeParams p) {
  pdl_sync();
  const GroupedShape& s = p.s;
  const int lane = threadIdx.x & 31;
  const long long item = blockIdx.x * 4ll + (threadIdx.x >> 5);
  if (item >= (long long)p.rows * s.heads) return;
  const int row = (int)(item / s.heads), h = (int)(item - (long long)row * s.heads);
  float gm[2] = {-INFINITY, -INFINITY}, inv[2] = {0.f, 0.f};
  const long long base = item * s.maps * p.splits;
#pragma unroll
  for (int mp = 0; mp < 2; ++mp) {
    if (mp >= s.maps) break;
    const float* ml = p.part_ml + (base + mp * p.splits) * 2;
    for (int i = 0; i < p.splits; ++i) gm[mp] = fmaxf(gm[mp], ml[i * 2]);
    float l = 0.f;
    for (int i = 0; i < p.splits; ++i) l += ml[i * 2] == -INFINITY ? 0.f : ml[i * 2 + 1] * exp2f(ml[i * 2] - gm[mp]);
    if (mp == 0 && s.sink != nullptr) add_sink(s.sink[h], gm[0], l);
    inv[mp] = l > 0.f ? 1.f / l : 0.f;
  }
  grouped_finish(s, lane, p.o + (long long)row * p.ld_o + h * s.vdim,
                 p.gate != nullptr ? p.gate + (long long)row * p.ld_gate + gate_column(s, h) : nullptr, [&](int mp, int c) {
                   const float* ml = p.part_ml + (base + mp * p.splits) * 2;
                   const float* po = p.part_o + (base + mp * p.splits) * s.vdim + c;
                   const float m = mp ? gm[1] : gm[0];
                   float v = 0.f;
                   for (int i = 0; i < p.splits; ++i)
                     if (ml[i * 2] != -INFINITY) v += po[(long long)i * s.vdim] * exp2f(ml[i * 2] - m);
                   return v * (mp ? inv[1] : inv[0]);
                 });
}

template <int KT, int VT>
static int launch_grouped_decode(const GroupedDecodeParams& p, cudaStream_t st) {
  constexpr int smem = GroupedDecodeSmem<KT, VT>::TOTAL;
  auto kern = grouped_decode_kernel<KT, VT>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
    configured = true;
  }
  launch_dep(kern, dim3(p.s.kv_heads * p.groups, p.rows, p.splits), GD_WARPS * 32, smem, st, p);
  if (p.splits > 1)
    launch_dep(grouped_merge_kernel, (unsigned)(((long long)p.rows * p.s.heads + 3) / 4), 128, 0, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_grouped_prep(const void* proj, long long ld, void* q, void* cache, const void* wq, const void* wk,
                                 const float* cos_sin, const int* positions, const long long* slots, int rows, int rot, int ctx,
                                 long long num_slots, const GroupedShape* s, int f32, uint32_t* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (!shape_ok(*s) || rot < 0 || rot > s->dim || (rot & 1) || (rot > 0 && cos_sin == nullptr) || wq == nullptr) return -10;
  GroupedPrepParams p;
  p.proj = proj; p.ld = ld; p.q = q; p.cache = cache; p.wq = wq; p.wk = wk; p.cos_sin = cos_sin; p.positions = positions;
  p.slots = slots; p.rows = rows; p.heads = s->heads; p.kv_heads = s->kv_heads; p.maps = s->maps; p.dim = s->dim;
  p.vdim = s->vdim; p.qp = s->qp; p.kp = s->kp; p.vp = s->vp; p.rot = rot; p.ctx = ctx; p.num_slots = num_slots;
  p.eps = s->eps; p.status = status;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) |
                         reinterpret_cast<uintptr_t>(wq) | reinterpret_cast<uintptr_t>(wk) | reinterpret_cast<uintptr_t>(cos_sin);
  if (s->dim % 8 == 0 && s->dim <= 256 && s->vdim % 8 == 0 && (rot / 2) % 8 == 0 && ld % 8 == 0 && (ptrs & 15) == 0) {
    if (f32) launch_prep_pieces<float>(p, st);
    else launch_prep_pieces<__nv_bfloat16>(p, st);
    return cudaGetLastError() == cudaSuccess ? 0 : -4;
  }
  const bool vec = s->dim % 4 == 0 && s->vdim % 4 == 0 && (rot / 2) % 4 == 0 && ld % 4 == 0 && (ptrs & 15) == 0;
  const long long items = (long long)rows * (s->heads * s->maps + (wk != nullptr ? s->kv_heads * (s->maps + 1) : 0));
  const int warps = items >= 148 * 8 * 4 ? 8 : 2;
  const unsigned grid = (unsigned)((items + warps - 1) / warps);
  if (f32) {
    if (vec) launch_dep(grouped_prep_kernel<float, 4>, grid, warps * 32, 0, st, p);
    else launch_dep(grouped_prep_kernel<float, 1>, grid, warps * 32, 0, st, p);
  } else {
    if (vec) launch_dep(grouped_prep_kernel<__nv_bfloat16, 4>, grid, warps * 32, 0, st, p);
    else launch_dep(grouped_prep_kernel<__nv_bfloat16, 1>, grid, warps * 32, 0, st, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// As b200_grouped_prep for one map, with one norm over all queries and one over all keys: wq (heads * dim), wk (kv_heads * dim).
extern "C" int b200_grouped_prep_whole(const void* proj, long long ld, void* q, void* cache, const void* wq, const void* wk,
                                       const float* cos_sin, const int* positions, const long long* slots, int rows, int rot, int ctx,
                                       long long num_slots, const GroupedShape* s, int f32, uint32_t* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (!shape_ok(*s) || s->maps != 1 || rot < 0 || rot > s->dim || (rot & 1) || (rot > 0 && cos_sin == nullptr) || wq == nullptr) return -10;
  GroupedPrepParams p;
  p.proj = proj; p.ld = ld; p.q = q; p.cache = cache; p.wq = wq; p.wk = wk; p.cos_sin = cos_sin; p.positions = positions;
  p.slots = slots; p.rows = rows; p.heads = s->heads; p.kv_heads = s->kv_heads; p.maps = 1; p.dim = s->dim;
  p.vdim = s->vdim; p.qp = s->qp; p.kp = s->kp; p.vp = s->vp; p.rot = rot; p.ctx = ctx; p.num_slots = num_slots;
  p.eps = s->eps; p.status = status;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) |
                         reinterpret_cast<uintptr_t>(wq) | reinterpret_cast<uintptr_t>(wk);
  const bool vec = s->dim % 8 == 0 && s->vdim % 8 == 0 && (rot / 2) % 8 == 0 && ld % 8 == 0 && (ptrs & 15) == 0;
  const int pieces = (s->heads * s->dim + (wk != nullptr ? s->kv_heads * (s->dim + s->vdim) : 0)) / (vec ? 8 : 1);
  int threads = ((pieces + 1) / 2 + 31) / 32 * 32;
  if (rows < 148 * 2) threads = (pieces + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const int lanes = s->dim / 8;
  const bool same = vec && lanes <= 32 && (lanes & (lanes - 1)) == 0 && (reinterpret_cast<uintptr_t>(cos_sin) & 15) == 0;
#define PREP_WHOLE(T)                                                                                  \
  if (same) launch_dep(grouped_prep_whole_pieces_kernel<T>, rows, threads, 0, st, p);                 \
  else if (vec) launch_dep(grouped_prep_whole_kernel<T, 8>, rows, threads, 0, st, p);                 \
  else launch_dep(grouped_prep_whole_kernel<T, 1>, rows, threads, 0, st, p)
  if (f32) {
    PREP_WHOLE(float);
  } else {
    PREP_WHOLE(__nv_bfloat16);
  }
#undef PREP_WHOLE
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

extern "C" int b200_grouped_rows(const void* q, const void* cache, void* o, long long ld_o, const void* gate, long long ld_gate,
                                 const float* bias, int bias_len, const int* row_seq, const int* positions,
                                 const long long* slots, const int* tables, int seqs, int rows, int max_pages, int page_size,
                                 int num_pages, const GroupedShape* s, int f32, uint32_t* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (!shape_ok(*s) || page_size <= 0 || (bias != nullptr && bias_len <= 0)) return -10;
  GroupedRowsParams p;
  p.q = q; p.cache = cache; p.o = o; p.ld_o = ld_o; p.gate = gate; p.ld_gate = ld_gate; p.bias = bias; p.bias_len = bias_len;
  p.row_seq = row_seq; p.positions = positions; p.slots = slots; p.tables = tables; p.seqs = seqs; p.rows = rows;
  p.max_pages = max_pages; p.page_size = page_size; p.num_pages = num_pages; p.s = *s; p.status = status;
  const size_t smem = 4ull * s->maps * (s->dim + s->vdim) * sizeof(float);
  if (smem > 200 * 1024) return -12;
  const unsigned grid = (unsigned)(((long long)rows * s->heads + 3) / 4);
  auto kern = f32 ? grouped_rows_kernel<float> : grouped_rows_kernel<__nv_bfloat16>;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return -3;
  launch_dep(kern, grid, 128, smem, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// bf16, one query row per line of the tables; maps * kp up to 256, vdim up to 128.  splits > 1 needs part_o (rows * heads * maps *
// splits * vdim floats) and part_ml (rows * heads * maps * splits * 2 floats).
extern "C" int b200_grouped_decode(const void* q, const void* cache, void* o, long long ld_o, const void* gate, long long ld_gate,
                                   const float* bias, int bias_len, float* part_o, float* part_ml, const int* positions,
                                   const long long* slots, const int* tables, int rows, int max_pages, int page_size,
                                   int num_pages, int splits, const GroupedShape* s, uint32_t* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  const int kd = s->maps * s->kp;
  if (!shape_ok(*s) || page_size <= 0 || kd > 256 || s->vp > 128 || splits < 1 || splits > 65535 || (bias != nullptr && bias_len <= 0))
    return -10;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15) return -10;
  if (splits > 1 && (part_o == nullptr || part_ml == nullptr)) return -11;
  GroupedDecodeParams p;
  p.q = (const __nv_bfloat16*)q; p.cache = (const __nv_bfloat16*)cache; p.gate = (const __nv_bfloat16*)gate;
  p.o = (__nv_bfloat16*)o; p.ld_o = ld_o; p.ld_gate = ld_gate; p.part_o = part_o; p.part_ml = part_ml; p.bias = bias;
  p.bias_len = bias_len; p.positions = positions; p.slots = slots; p.tables = tables; p.rows = rows; p.max_pages = max_pages;
  p.page_size = page_size; p.num_pages = num_pages; p.splits = splits; p.s = *s; p.status = status;
  const int hpg = 16 / s->maps;
  p.groups = (s->heads / s->kv_heads + hpg - 1) / hpg;
  if (rows > 65535) return -12;
  const bool v64 = s->vp <= 64;
  if (kd <= 64) return v64 ? launch_grouped_decode<4, 8>(p, st) : launch_grouped_decode<4, 16>(p, st);
  if (kd <= 128) return v64 ? launch_grouped_decode<8, 8>(p, st) : launch_grouped_decode<8, 16>(p, st);
  return v64 ? launch_grouped_decode<16, 8>(p, st) : launch_grouped_decode<16, 16>(p, st);
}
