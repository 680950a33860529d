// Gated delta rule.  Per head, with a decay g_t in (0, 1), a write strength beta_t in (0, 1) and unit vectors k_t, q_t:
//     S <- g_t S,   u = beta_t (v_t - S^T k_t),   S <- S + k_t u^T,   o_t = S^T q_t
// then o_t / rms(o_t) * weight * silu(gate).  q_t = q / |q| * dim^(-1/2) and k_t = k / |k| (|x|^2 = sum x^2 + 1e-6); heads / kv_heads heads
// share a q and a k.  log g_t = -exp(A) softplus(a_t + dt), beta_t = sigmoid(b_t); a and b arrive in fp32.  q, k, v have passed a short
// convolution and silu (short_conv.cu; the fused decode step does that itself).  The state S (dim, vdim) is fp32 and lives in a slot.
//
// q and k enter products as they are stored; their inverse lengths, the decays and beta are fp32 factors of what comes out.
#include "typed.cuh"

namespace b200 {

int make_tmap_bf16_2d(CUtensorMap* tm, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_cols,
                      uint32_t box_rows);

// Passed by pointer through the C interface: the field order is part of it.
struct DeltaArgs {
  const void* c;             // (rows, ld_c): q (kv_heads, dim) | k (kv_heads, dim) | v (heads, vdim); before the convolution if taps > 0
  const void* gate;          // (rows, ld_gate): (heads, vdim)
  const float* ab;           // (rows, ld_ab): a of all heads | b of all heads; null: products of h and w_ab, taken here
  const void *h, *w_ab;      // (rows, ld_h), (2 * heads, ld_w): `width` columns
  const float *decay, *dt;   // (heads): -exp(A), dt
  const void* weight;        // (vdim)
  const void* filter;        // (taps, channels)
  void* ring;                // (num_slots, taps, channels)
  void* y;                   // (rows, ld_y)
  float* state;              // (num_slots, heads, dim, vdim)
  void* image;               // chunked: a piece per chunk and head
  const int *state_slots, *cu, *positions, *chunk_cu;    // cu (seqs + 1): rows; chunk_cu (seqs + 1): chunks of each sequence
  uint32_t* status;
  long long ld_c, ld_gate, ld_ab, ld_h, ld_w, ld_y;
  int width, taps, seqs, rows, heads, kv_heads, dim, vdim, num_slots, chunks;
  float eps;
};

__device__ __forceinline__ float delta_log_decay(float z, float decay) {      // decay <= 0
  return decay * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))));
}

// One block per (sequence, head), tokens in order, the state in global memory (every thread re-reads only what it wrote): any sizes,
// T = bf16 or fp32.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) delta_recurrent_kernel(const DeltaArgs p) {
  pdl_sync();
  extern __shared__ float dsm[];
  __shared__ float red[32];
  const int seq = blockIdx.x, h = blockIdx.y, D = p.dim, E = p.vdim, hk = h / (p.heads / p.kv_heads);
  const int groups = E / VEC, cgt = groups < 256 ? groups : 256, rg = 256 / cgt;
  float *qs = dsm, *ks = qs + D, *us = ks + D, *pk = us + E, *pq = pk + rg * E;      // [D], [D], [E], [rg][E], [rg][E]
  const int ty = threadIdx.x / cgt, tx = threadIdx.x - ty * cgt;
  const int row0 = p.cu != nullptr ? p.cu[seq] : seq, row1 = p.cu != nullptr ? p.cu[seq + 1] : seq + 1;
  const int slot = p.state_slots[seq];
  T* y = reinterpret_cast<T*>(p.y);
  if (slot < 0 || slot >= p.num_slots) {
    if (slot >= p.num_slots && threadIdx.x == 0) report_bad_arg(p.status, 50);
    for (int row = row0; row < row1; ++row)
      for (int c = threadIdx.x; c < E; c += 256) from_f(y[(long long)row * p.ld_y + h * E + c], 0.f);
    return;
  }
  float* S = p.state + ((long long)slot * p.heads + h) * D * E;
  for (int row = row0; row < row1; ++row) {
    const bool fresh = p.positions[row] == 0;        // a sequence starts from the zero state, whatever its slot held
    const T* cr = reinterpret_cast<const T*>(p.c) + (long long)row * p.ld_c;
    const T *qr = cr + hk * D, *kr = cr + (p.kv_heads + hk) * D, *vr = cr + 2 * p.kv_heads * D + h * E;
    const float* ab = p.ab + (long long)row * p.ld_ab;
    const float g = expf(delta_log_decay(ab[h] + p.dt[h], p.decay[h])), beta = 1.f / (1.f + expf(-ab[p.heads + h]));
    float qq = 0.f, kk = 0.f, kq = 0.f;
    for (int d = threadIdx.x; d < D; d += 256) {
      const float a = to_f(qr[d]), b = to_f(kr[d]);
      qs[d] = a;
      ks[d] = b;
      qq = fmaf(a, a, qq);
      kk = fmaf(b, b, kk);
      kq = fmaf(a, b, kq);
    }
    qq = block_total(qq, red);                       // the barriers also publish qs and ks
    kk = block_total(kk, red);
    kq = block_total(kq, red);
    const float iq = rsqrtf(qq + 1e-6f) * rsqrtf((float)D), ik = rsqrtf(kk + 1e-6f);
    if (ty < rg) {
      for (int gr = tx; gr < groups; gr += cgt) {
        float ak[VEC], aq[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) ak[i] = aq[i] = 0.f;
        if (!fresh) {
#pragma unroll 4
          for (int d = ty; d < D; d += rg) {
            float s[VEC];
            load_vec<VEC>(S + (long long)d * E + gr * VEC, s);
            const float kd = ks[d], qd = qs[d];
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
              ak[i] = fmaf(s[i], kd, ak[i]);
              aq[i] = fmaf(s[i], qd, aq[i]);
            }
          }
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          pk[ty * E + gr * VEC + i] = ak[i];
          pq[ty * E + gr * VEC + i] = aq[i];
        }
      }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = threadIdx.x; c < E; c += 256) {
      float sk = 0.f, sq = 0.f;
      for (int r = 0; r < rg; ++r) {
        sk += pk[r * E + c];
        sq += pq[r * E + c];
      }
      const float u = beta * (to_f(vr[c]) - g * ik * sk);
      const float o = iq * fmaf(g, sq, kq * ik * u);
      us[c] = u;
      pq[c] = o;                                     // row 0 of this column is read by this thread only
      ss = fmaf(o, o, ss);
    }
    const float inv = rsqrtf(block_total(ss, red) / (float)E + p.eps);      // its barriers also publish us
    if (ty < rg) {
      for (int gr = tx; gr < groups; gr += cgt) {
        float u[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] = us[gr * VEC + i] * ik;
#pragma unroll 4
        for (int d = ty; d < D; d += rg) {
          float s[VEC];
          float* sp = S + (long long)d * E + gr * VEC;
          if (fresh) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) s[i] = 0.f;
          } else {
            load_vec<VEC>(sp, s);
          }
          const float kd = ks[d];
#pragma unroll
          for (int i = 0; i < VEC; ++i) s[i] = fmaf(g, s[i], kd * u[i]);
          store_vec<VEC>(sp, s);
        }
      }
    }
    const T* w = reinterpret_cast<const T*>(p.weight);
    const T* gr = reinterpret_cast<const T*>(p.gate) + (long long)row * p.ld_gate + h * E;
    for (int c = threadIdx.x; c < E; c += 256) {
      const float z = to_f(gr[c]);
      from_f(y[(long long)row * p.ld_y + h * E + c], pq[c] * inv * to_f(w[c]) * z / (1.f + expf(-z)));
    }
    __syncthreads();
  }
}

// Decode step of a state that fits the block's registers (NR rows of four columns per thread): one block per (request, head); the
// whole state is requested before anything else, so the convolution, the lengths and the gates run under its latency.  S^T k and S^T q of
// the old state come from one pass; the new output is g S^T q + (k . q) u.
template <typename T, int NR>
__global__ void __launch_bounds__(256, NR > 8 ? 2 : 3) delta_step_kernel(const DeltaArgs p) {
  pdl_sync();
  extern __shared__ float dsm[];
  __shared__ float red[5][8];
  const int seq = blockIdx.x / p.heads, h = blockIdx.x - seq * p.heads;
  const int D = p.dim, E = p.vdim, groups = E / 4, rg = 256 / groups, rep = p.heads / p.kv_heads, hk = h / rep;
  float *qs = dsm, *ks = qs + D, *vs = ks + D, *us = vs + E;
  float *pk = dsm + (2 * D + 2 * E + 3) / 4 * 4, *pq = pk + rg * E;                  // [rg][E] each
  const int ty = threadIdx.x / groups, tx = threadIdx.x - ty * groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slot = p.state_slots[seq];
  T* y = reinterpret_cast<T*>(p.y) + (long long)seq * p.ld_y + h * E;
  if (slot < 0 || slot >= p.num_slots) {
    if (slot >= p.num_slots && threadIdx.x == 0) report_bad_arg(p.status, 51);
    for (int c = threadIdx.x; c < E; c += 256) from_f(y[c], 0.f);
    return;
  }
  const int pos = p.positions[seq];
  const bool fresh = pos == 0, on = ty < rg;
  float4* S = reinterpret_cast<float4*>(p.state + ((long long)slot * p.heads + h) * D * E) + tx;
  // the operands of the gates are few and in L2: the first of them are requested before the state, not behind it
  float hx[4] = {0.f, 0.f, 0.f, 0.f}, ha[4] = {0.f, 0.f, 0.f, 0.f}, hb[4] = {0.f, 0.f, 0.f, 0.f};
  const T* hr = reinterpret_cast<const T*>(p.h) + (long long)seq * p.ld_h;
  const T* wa = reinterpret_cast<const T*>(p.w_ab) + (long long)h * p.ld_w;
  const T* wb = wa + (long long)p.heads * p.ld_w;
  if (p.ab == nullptr && threadIdx.x * 4 < p.width) {
    load_vec<4>(hr + threadIdx.x * 4, hx);
    load_vec<4>(wa + threadIdx.x * 4, ha);
    load_vec<4>(wb + threadIdx.x * 4, hb);
  }
  // q, k, v of this head, 2 D + E channels: those of a thread's first two, with up to four taps, are requested before the state as well
  const T* cr = reinterpret_cast<const T*>(p.c) + (long long)seq * p.ld_c;
  const int channels = 2 * p.kv_heads * D + p.heads * E, mine_n = 2 * D + E;
  const T* filter = reinterpret_cast<const T*>(p.filter);
  T* ring = reinterpret_cast<T*>(p.ring) + (long long)slot * p.taps * channels;
  auto channel = [&](int i) {
    return i < D ? hk * D + i : (i < 2 * D ? (p.kv_heads + hk) * D + i - D : 2 * p.kv_heads * D + h * E + i - 2 * D);
  };
  constexpr int AHEAD = 2, TAPS = 4;
  T raw[AHEAD], past[AHEAD][TAPS], weight[AHEAD][TAPS];
#pragma unroll
  for (int k = 0; k < AHEAD; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i >= mine_n) break;
    const int ch = channel(i);
    raw[k] = cr[ch];
#pragma unroll
    for (int d = 0; d < TAPS; ++d) {
      from_f(past[k][d], 0.f);
      if (d < p.taps) weight[k][d] = filter[(long long)(p.taps - 1 - d) * channels + ch];
      if (d > 0 && d < p.taps && pos >= d) past[k][d] = ring[(long long)((pos - d) % p.taps) * channels + ch];
    }
  }
  const T* gr = reinterpret_cast<const T*>(p.gate) + (long long)seq * p.ld_gate + h * E;
  const float z0 = threadIdx.x < E ? to_f(gr[threadIdx.x]) : 0.f, w0 = threadIdx.x < E ? to_f(reinterpret_cast<const T*>(p.weight)[threadIdx.x]) : 0.f;
  float4 s[NR];
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = ty + j * rg;
    s[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on && d < D && !fresh) s[j] = __ldcs(S + (long long)d * groups);
  }
  float qq = 0.f, kk = 0.f;
  auto place = [&](int i, T now, float f) {                // f: the convolution, or the channel itself
    if (p.taps > 0) {
      if (i >= 2 * D || h == hk * rep) ring[(long long)(pos % p.taps) * channels + channel(i)] = now;      // nobody reads this row in this step
      f = f / (1.f + expf(-f));
    }
    qs[i] = f;                                       // qs | ks | vs
  };
#pragma unroll
  for (int k = 0; k < AHEAD; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i >= mine_n || p.taps > TAPS) break;
    float f = to_f(raw[k]);
    if (p.taps > 0) f *= to_f(weight[k][0]);
#pragma unroll
    for (int d = 1; d < TAPS; ++d)
      if (d < p.taps) f = fmaf(to_f(weight[k][d]), to_f(past[k][d]), f);
    place(i, raw[k], f);
  }
  for (int i = threadIdx.x + (p.taps > TAPS ? 0 : AHEAD * 256); i < mine_n; i += 256) {
    const int ch = channel(i);
    const T now = cr[ch];
    float f = to_f(now);
    if (p.taps > 0) f *= to_f(filter[(long long)(p.taps - 1) * channels + ch]);
    for (int d = 1; d < p.taps; ++d)
      if (pos >= d) f = fmaf(to_f(filter[(long long)(p.taps - 1 - d) * channels + ch]), to_f(ring[(long long)((pos - d) % p.taps) * channels + ch]), f);
    place(i, now, f);
  }
  float za = 0.f, zb = 0.f;
  if (p.ab != nullptr) {
    if (threadIdx.x == 0) {
      za = p.ab[(long long)seq * p.ld_ab + h];
      zb = p.ab[(long long)seq * p.ld_ab + p.heads + h];
    }
  } else {
    for (int c = threadIdx.x * 4; c < p.width; c += 1024) {            // pitches are multiples of 4, what lies in the pads is left out
      if (c >= 1024) {
        load_vec<4>(hr + c, hx);
        load_vec<4>(wa + c, ha);
        load_vec<4>(wb + c, hb);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float xv = c + i < p.width ? hx[i] : 0.f;
        za = fmaf(xv, ha[i], za);
        zb = fmaf(xv, hb[i], zb);
      }
    }
  }
  __syncthreads();                                   // q, k, v are there
  float kq = 0.f;
  for (int d = threadIdx.x; d < D; d += 256) {
    const float a = qs[d], b = ks[d];
    qq = fmaf(a, a, qq);
    kk = fmaf(b, b, kk);
    kq = fmaf(a, b, kq);
  }
  // five sums over the block at once
  float sums[5] = {qq, kk, kq, za, zb};
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int i = 0; i < 5; ++i) sums[i] += __shfl_xor_sync(0xffffffffu, sums[i], o);
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < 5; ++i) red[i][warp] = sums[i];
  }
  float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = ty + j * rg;
    if (!on || d >= D) continue;
    const float kd = ks[d], qd = qs[d];
    ak.x = fmaf(s[j].x, kd, ak.x); ak.y = fmaf(s[j].y, kd, ak.y); ak.z = fmaf(s[j].z, kd, ak.z); ak.w = fmaf(s[j].w, kd, ak.w);
    aq.x = fmaf(s[j].x, qd, aq.x); aq.y = fmaf(s[j].y, qd, aq.y); aq.z = fmaf(s[j].z, qd, aq.z); aq.w = fmaf(s[j].w, qd, aq.w);
  }
  if (on) {
    *reinterpret_cast<float4*>(pk + ty * E + tx * 4) = ak;
    *reinterpret_cast<float4*>(pq + ty * E + tx * 4) = aq;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 5; ++i) {
    sums[i] = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) sums[i] += red[i][w];
  }
  const float iq = rsqrtf(sums[0] + 1e-6f) * rsqrtf((float)D), ik = rsqrtf(sums[1] + 1e-6f);
  const float g = expf(delta_log_decay(sums[3] + p.dt[h], p.decay[h])), beta = 1.f / (1.f + expf(-sums[4]));
  float ss = 0.f, mine[4];
  int n = 0;
  for (int c = threadIdx.x; c < E && n < 4; c += 256, ++n) {           // E <= 1024
    float sk = 0.f, sq = 0.f;
    for (int r = 0; r < rg; ++r) {
      sk += pk[r * E + c];
      sq += pq[r * E + c];
    }
    const float u = beta * (vs[c] - g * ik * sk);
    us[c] = u * ik;
    mine[n] = iq * fmaf(g, sq, sums[2] * ik * u);
    ss = fmaf(mine[n], mine[n], ss);
  }
  const float inv = rsqrtf(block_total(ss, red[0]) / (float)E + p.eps);      // its barriers also publish us
  if (on) {
    const float4 u = make_float4(us[tx * 4], us[tx * 4 + 1], us[tx * 4 + 2], us[tx * 4 + 3]);
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int d = ty + j * rg;
      if (d >= D) continue;
      const float kd = ks[d];
      s[j].x = fmaf(g, s[j].x, kd * u.x); s[j].y = fmaf(g, s[j].y, kd * u.y);
      s[j].z = fmaf(g, s[j].z, kd * u.z); s[j].w = fmaf(g, s[j].w, kd * u.w);
      __stcs(S + (long long)d * groups, s[j]);
    }
  }
  n = 0;
  for (int c = threadIdx.x; c < E && n < 4; c += 256, ++n) {
    const float z = n == 0 ? z0 : to_f(gr[c]), w = n == 0 ? w0 : to_f(reinterpret_cast<const T*>(p.weight)[c]);
    from_f(y[c], mine[n] * inv * w * z * sigmoid_f(z));
  }
}

// ------------------------------------------------------------------------------------ prompts, bf16, on the tensor cores
// Chunks of 64 tokens.  Inside a chunk let b_t = log g_1 + ... + log g_t.  With S the state before the chunk, the writes u_t solve
//     u_t + sum_(s < t) A_ts u_s = beta_t (v_t - exp(b_t) S^T k_t),      A_ts = beta_t exp(b_t - b_s) k_t . k_s
// and o_t = exp(b_t) S^T q_t + sum_(s <= t) P_ts u_s with P_ts = exp(b_t - b_s) q_t . k_s,  S <- exp(b_n) S + sum_s exp(b_n - b_s) k_s u_s^T.
// Every exponent is at most zero.  T = (I + A)^-1 does not depend on S:
//   delta_prepare   all chunks at once, one CTA each: scores and squared lengths of [K; Q] on tcgen05, T in fp32 by forward substitution of its diagonal
//                   blocks and products, T and P split into two bf16 parts (hi + lo, 16 significant bits), the per-token factors: an image of 33 KB
//                   that the second kernel copies as it is
//   delta_chunk     one CTA per (portion, head), chunks in order, everything transposed so that a lane of tensor memory is a column of v:
//                     V^T (a product with the unit matrix)  [S^T K^T | S^T Q^T]  ->  R = beta (V - ...)^T  ->  U^T = R T^T  ->  S^T = exp(b_n) S^T + W K,  P U  (W: U with its factors)
//                   S, R, U and W are A operands in tensor memory, split like T and P; products accumulate in fp32 (lo x lo is dropped)
constexpr int DC = 64;                              // tokens of a chunk
constexpr int DC_TILE = DC * 128;                   // bytes of 64 rows of 64 bf16 columns, 128-byte swizzle
constexpr int DI_T = 0, DI_P = 2 * DC_TILE, DI_F = 4 * DC_TILE;      // image: T hi, lo | P hi, lo | (beta, -beta c), w, a per token | exp(b_n)
constexpr int DI_BYTES = DI_F + 4 * DC * 4 + 128;
constexpr float DELTA_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float dl_exp2(float x) {       // x <= 0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float dl_sigmoid(float g) {    // (1 + tanh(g / 2)) / 2
  float t;
  asm("tanh.approx.f32 %0, %1;" : "=f"(t) : "f"(0.5f * g));
  return fmaf(0.5f, t, 0.5f);
}
// Two values as hi + lo, both bf16: hi is cut off (the remainder is exact), lo rounded.
__device__ __forceinline__ void dl_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const uint32_t a = __float_as_uint(x), b = __float_as_uint(y);
  hi = __byte_perm(a, b, 0x7632);
  lo = pack_bf16x2(x - __uint_as_float(a & 0xffff0000u), y - __uint_as_float(b & 0xffff0000u));
}
__device__ __forceinline__ uint32_t dl_swz(int r, int c8) { return (uint32_t)r * 128u + (uint32_t)((c8 ^ (r & 7)) << 4); }

constexpr int DP_HEADS = 2;                         // heads with the same keys that a CTA takes, one after the other
struct DeltaPrepareSmem {                           // X: panels of [64 rows of K; 64 rows of Q] x 64 columns, later the image
  static constexpr int OFF_X = 0, OFF_I = 0, OFF_A = (DI_BYTES + 1023) / 1024 * 1024;
  static constexpr int PITCH = 68;                  // floats between the rows of A
  static constexpr int OFF_F = OFF_A + DC * PITCH * 4;        // b [64], beta [64], inverse lengths [128]
  static constexpr int OFF_BAR = OFF_F + 4 * DC * 4;
  static constexpr int TOTAL = OFF_BAR + 2 * 8 + 16 + 1024;
};

__global__ void __launch_bounds__(128) delta_prepare_kernel(const __grid_constant__ CUtensorMap tm, const DeltaArgs p) {
  using L = DeltaPrepareSmem;
  extern __shared__ uint8_t dl_raw[];
  uint8_t* smem = dl_raw + (-smem_u32(dl_raw) & 1023u);        // (an offset, so that accesses stay known as shared)
  float* A = reinterpret_cast<float*>(smem + L::OFF_A);
  auto at = [&](int row, int col) { return A + row * L::PITCH + col; };
  float *sb = reinterpret_cast<float*>(smem + L::OFF_F), *sbeta = sb + DC, *slen = sbeta + DC;
  uint64_t *bar_l = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR), *bar_m = bar_l + 1;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bar_l + 2);
  volatile uint32_t* abort_word = tmem_holder + 1;
  __shared__ float half_sum;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    mbar_init(bar_l, 1);
    mbar_init(bar_m, 1);
    *abort_word = 0;
    fence_barrier_init();
    prefetch_tensormap(&tm);
  }
  if (warp == 0) {
    tmem_alloc(tmem_holder, 128);
    tmem_relinquish();
  }
  pdl_sync();
  const int rep = p.heads / p.kv_heads, sets = (rep + DP_HEADS - 1) / DP_HEADS, set = blockIdx.x % sets;
  const int hk = blockIdx.x / sets % p.kv_heads, chunk = blockIdx.x / (sets * p.kv_heads), D = p.dim;
  const int h0 = hk * rep + set * DP_HEADS, heads = min(DP_HEADS, rep - set * DP_HEADS);      // heads h0 .. share these keys
  int lo = 0, hi = p.seqs;                          // the portion the chunk belongs to
  while (hi - lo > 1) {
    const int mid = (lo + hi) / 2;
    if (p.chunk_cu[mid] <= chunk) lo = mid;
    else hi = mid;
  }
  const int row0 = p.cu[lo] + (chunk - p.chunk_cu[lo]) * DC, n = min(DC, p.cu[lo + 1] - row0);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;
  const int pd = (D + 63) / 64, ksteps = (D + 15) / 16;
  if (tid == 0) {
    mbar_expect_tx(bar_l, (uint32_t)(2 * pd) * DC_TILE);
    for (int i = 0; i < pd; ++i) {
      tma_load_2d(smem + L::OFF_X + i * 16384, &tm, bar_l, (p.kv_heads + hk) * D + i * 64, row0);
      tma_load_2d(smem + L::OFF_X + i * 16384 + DC_TILE, &tm, bar_l, hk * D + i * 64, row0);
    }
  }
  // ---- decays, added up over each half of the tokens, and write strengths; tokens that are not there neither decay nor write
  auto gates = [&](int h) {
    float b = 0.f, beta = 0.f;
    if (tid < n) {
      const float* ab = p.ab + (long long)(row0 + tid) * p.ld_ab;
      b = delta_log_decay(ab[h] + p.dt[h], p.decay[h]) * DELTA_LOG2E;
      beta = 1.f / (1.f + expf(-ab[p.heads + h]));
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, b, o);
      if (lane >= o) b += x;
    }
    if (tid == 31) half_sum = b;
    sbeta[tid] = beta;
    return b;
  };
  float b = tid < DC ? gates(h0) : 0.f;
  bool ok = mbar_wait(bar_l, 0, abort_word);
  if (!ok) *abort_word = ERR_WAIT_FULL;
  const int r = tid;                                // row of X
  if (D & 15) *reinterpret_cast<uint4*>(smem + L::OFF_X + (D >> 6) * 16384 + dl_swz(r, (D >> 3) & 7)) = make_uint4(0, 0, 0, 0);
  fence_proxy_async_smem();
  __syncthreads();
  if (warp == 0 && elect_one()) {
    constexpr uint32_t id = make_idesc_bf16(128, 128, false, false);
    const uint64_t x = make_smem_desc(smem_u32(smem + L::OFF_X), 16, 1024);
    for (int k = 0; k < ksteps; ++k) {
      const uint32_t off = ((k / 4) * 16384 + (k % 4) * 32) >> 4;
      umma_f16_ss(tmem, x + off, x + off, id, k ? 1u : 0u);
    }
    umma_commit(bar_m);
  }
  ok = mbar_wait(bar_m, 0, abort_word) && ok;
  if (!ok) *abort_word = ERR_WAIT_MISC;
  tc_fence_after();
  {                                                 // the diagonal: squared lengths
    uint32_t raw[32];
    tmem_ld_32x32(tmem + (uint32_t(warp * 32) << 16) + warp * 32, raw);
    tmem_ld_wait();
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 32; ++i) ss = i == lane ? __uint_as_float(raw[i]) : ss;
    slen[r] = rsqrtf(ss + 1e-6f) * (r < DC ? 1.f : rsqrtf((float)D));
  }
  const int t = r & (DC - 1);
  uint8_t* image = smem + L::OFF_I;
#pragma unroll 1
  for (int head = 0; head < heads; ++head) {
    if (head > 0) {
      if (tid == 0) tma_store_wait_read<0>();
      __syncthreads();                                // the image of the head before has left
      if (tid < DC) b = gates(h0 + head);
      __syncthreads();
    }
    if (tid < DC) sb[tid] = tid >= 32 ? b + half_sum : b;
    __syncthreads();
    const float bt = sb[t], mine = slen[r] * (r < DC ? sbeta[t] : 1.f);
    const int last = r < DC ? t - 1 : t;              // A lies strictly below the diagonal
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const bool any = half == 0 || (warp & 1) == 1;  // the first 32 tokens see none of the others
      uint32_t raw[32];
      if (any) {
        tmem_ld_32x32(tmem + (uint32_t(warp * 32) << 16) + half * 32, raw);
        tmem_ld_wait();
      } else if (r < DC) {
        continue;                                     // (that part of A is not read)
      }
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        float f[8];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int s = half * 32 + q * 8 + j * 4;
          float4 lens = make_float4(0.f, 0.f, 0.f, 0.f), bs = lens;
          if (any) {
            lens = *reinterpret_cast<const float4*>(slen + s);
            bs = *reinterpret_cast<const float4*>(sb + s);
          }
          const float l4[4] = {lens.x, lens.y, lens.z, lens.w}, b4[4] = {bs.x, bs.y, bs.z, bs.w};
#pragma unroll
          for (int i = 0; i < 4; ++i)
            f[j * 4 + i] = any && s + i <= last ? __uint_as_float(raw[q * 8 + j * 4 + i]) * (mine * l4[i]) * dl_exp2(fminf(bt - b4[i], 0.f)) : 0.f;
        }
        if (r < DC) {
          *reinterpret_cast<float4*>(at(t, half * 32 + q * 8)) = make_float4(f[0], f[1], f[2], f[3]);
          *reinterpret_cast<float4*>(at(t, half * 32 + q * 8 + 4)) = make_float4(f[4], f[5], f[6], f[7]);
        } else {
          uint4 hi4, lo4;
          dl_split2(f[0], f[1], hi4.x, lo4.x);
          dl_split2(f[2], f[3], hi4.y, lo4.y);
          dl_split2(f[4], f[5], hi4.z, lo4.z);
          dl_split2(f[6], f[7], hi4.w, lo4.w);
          *reinterpret_cast<uint4*>(image + DI_P + dl_swz(t, half * 4 + q)) = hi4;
          *reinterpret_cast<uint4*>(image + DI_P + DC_TILE + dl_swz(t, half * 4 + q)) = lo4;
        }
      }
    }
    tc_fence_before();
    __syncthreads();
    // ---- T from its diagonal blocks of 16 (forward substitution, a warp per block, a lane per column), then twice
    // T21 = -T22 (A21 T11), for blocks of 16 and of 32.  Products are kept above the diagonal, where A has nothing.
    constexpr int HB = DC / 2, QB = DC / 4;
    {
      const int o = warp * QB, c = lane & (QB - 1);
      float x[QB];
#pragma unroll
      for (int i = 0; i < QB; ++i) {
        float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int s = 0; s < i; s += 4) {
          const float4 v = *reinterpret_cast<const float4*>(at(o + i, o + s));
          a[0] = fmaf(v.x, x[s], a[0]);
          if (s + 1 < i) a[1] = fmaf(v.y, x[s + 1], a[1]);
          if (s + 2 < i) a[2] = fmaf(v.z, x[s + 2], a[2]);
          if (s + 3 < i) a[3] = fmaf(v.w, x[s + 3], a[3]);
        }
        x[i] = (i == c ? 1.f : 0.f) - ((a[0] + a[1]) + (a[2] + a[3]));
      }
      __syncwarp();                                   // the block has been read
      if (lane < QB) {
#pragma unroll
        for (int i = 0; i < QB; ++i) *at(o + i, o + c) = x[i];
      }
    }
    if (r >= DC) {
      float* f = reinterpret_cast<float*>(image + DI_F);
      const float end = sb[DC - 1], grown = dl_exp2(bt);
      *reinterpret_cast<float2*>(f + 2 * t) = make_float2(sbeta[t], -sbeta[t] * grown * slen[t]);      // of v_t, of S^T k_t
      f[2 * DC + t] = dl_exp2(end - bt) * slen[t];    // of u_t where it joins the state
      f[3 * DC + t] = grown * slen[r];                // of S^T q_t
      if (t == 0) f[4 * DC] = dl_exp2(end);
    }
    __syncthreads();
    {
      // two pairs of blocks, two warps each: 8 rows of a 16 x 16 product per warp, four of them per half warp
      const int o = (warp >> 1) * HB, c = lane & (QB - 1), i0 = (warp & 1) * 8 + (lane >> 4) * 4;
      auto small = [&](int lr, int lc, int rr, int rc, float (&acc)[4]) __attribute__((always_inline)) {
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i] = 0.f;
#pragma unroll
        for (int s = 0; s < QB; s += 4) {
          float v[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) v[j] = *at(rr + s + j, rc + c);
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float4 w = *reinterpret_cast<const float4*>(at(lr + i0 + i, lc + s));
            acc[i] = fmaf(w.x, v[0], fmaf(w.y, v[1], fmaf(w.z, v[2], fmaf(w.w, v[3], acc[i]))));
          }
        }
      };
      float acc[4];
      small(o + QB, o, o, o, acc);
#pragma unroll
      for (int i = 0; i < 4; ++i) *at(o + i0 + i, o + QB + c) = acc[i];
      __syncthreads();
      small(o + QB, o + QB, o, o + QB, acc);
#pragma unroll
      for (int i = 0; i < 4; ++i) *at(o + QB + i0 + i, o + c) = -acc[i];
      __syncthreads();
#pragma unroll
      for (int i = 0; i < 4; ++i) *at(o + i0 + i, o + QB + c) = 0.f;
    }
    __syncthreads();
    // rows warp * 8 .. + 7 and column `lane` of the product of the blocks at (lr, lc) and (rr, rc)
    auto product = [&](int lr, int lc, int rr, int rc, float (&acc)[8]) __attribute__((always_inline)) {
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i] = 0.f;
#pragma unroll
      for (int s = 0; s < HB; s += 4) {
        float v[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) v[j] = *at(rr + s + j, rc + lane);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float4 w = *reinterpret_cast<const float4*>(at(lr + warp * 8 + i, lc + s));
          acc[i] = fmaf(w.x, v[0], fmaf(w.y, v[1], fmaf(w.z, v[2], fmaf(w.w, v[3], acc[i]))));
        }
      }
    };
    float acc[8];
    product(HB, 0, 0, 0, acc);               // A21 T11, kept above the diagonal
#pragma unroll
    for (int i = 0; i < 8; ++i) *at(warp * 8 + i, HB + lane) = acc[i];
    __syncthreads();
    product(HB, HB, 0, HB, acc);
#pragma unroll
    for (int i = 0; i < 8; ++i) *at(HB + warp * 8 + i, lane) = -acc[i];
    __syncthreads();
    {
      const int row = r >> 1, half = r & 1;
      const bool zero = row < HB && half == 1;        // above the diagonal
      float4 u[8];
#pragma unroll
      for (int q = 0; q < 8; ++q) u[q] = zero ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(at(row, half * 32 + q * 4));
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        uint4 hi4, lo4;
        dl_split2(u[2 * q].x, u[2 * q].y, hi4.x, lo4.x);
        dl_split2(u[2 * q].z, u[2 * q].w, hi4.y, lo4.y);
        dl_split2(u[2 * q + 1].x, u[2 * q + 1].y, hi4.z, lo4.z);
        dl_split2(u[2 * q + 1].z, u[2 * q + 1].w, hi4.w, lo4.w);
        *reinterpret_cast<uint4*>(image + DI_T + dl_swz(row, half * 4 + q)) = hi4;
        *reinterpret_cast<uint4*>(image + DI_T + DC_TILE + dl_swz(row, half * 4 + q)) = lo4;
      }
    }
    fence_proxy_async_smem();
    __syncthreads();
    if (tid == 0) {
      uint8_t* to = reinterpret_cast<uint8_t*>(p.image) + ((long long)chunk * p.heads + h0 + head) * DI_BYTES;
      asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(reinterpret_cast<uint64_t>(to)), "r"(smem_u32(image)),
                   "r"((uint32_t)DI_BYTES)
                   : "memory");
      tma_store_commit();
    }
  }
  if (tid == 0) {
    tma_store_wait<0>();
    if (*abort_word != 0 && p.status != nullptr) atomicCAS(p.status, 0u, (*abort_word) | (blockIdx.x << 8));
  }
  tc_fence_before();
  __syncthreads();
  if (*abort_word != 0) {                           // give copies that may still be in flight time to land
    const uint64_t w0 = globaltimer_ns();
    while (globaltimer_ns() - w0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(tmem, 128);
  }
}

// Warps 0 - 7: the chain R, U, S (a lane of tensor memory and half of the columns per thread); 8 - 15: outputs; 16: copies; 17: products.
constexpr int DK_CHAIN = 8, DK_OUT = 8, DK_THREADS = (DK_CHAIN + DK_OUT + 2) * 32;

template <int PD, int PE>                            // panels of 64 columns of q and k, and of v
struct DeltaChunkSmem {
  static constexpr int X = PD * 16384, V = PE * DC_TILE, I = (DI_BYTES + 1023) / 1024 * 1024, STAGE = X + V + I;
  static constexpr int OFF_O = 2 * STAGE;            // [64][PE * 64] floats
  static constexpr int OFF_G = OFF_O + DC * PE * 64 * 4;       // output gates
  static constexpr int OFF_ONE = OFF_G + PE * DC_TILE;         // the unit matrix, bf16
  static constexpr int OFF_BAR = OFF_ONE + DC_TILE;
  static constexpr int NUM_BARS = 14;
  static constexpr int TOTAL = OFF_BAR + NUM_BARS * 8 + 16 + 1024;
};

template <int PD, int PE>
__global__ void __launch_bounds__(DK_THREADS, 1) delta_chunk_kernel(const __grid_constant__ CUtensorMap tm,
                                                                     const __grid_constant__ CUtensorMap tm_gate, const DeltaArgs p) {
  using L = DeltaChunkSmem<PD, PE>;
  extern __shared__ uint8_t dl_raw[];
  uint8_t* smem = dl_raw + (-smem_u32(dl_raw) & 1023u);        // (an offset, so that accesses stay known as shared)
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR);
  uint64_t *full = bars, *empty = bars + 2;          // [2] per stage
  uint64_t *s_ready = bars + 4, *d1_full = bars + 5, *r_ready = bars + 6, *d2_full = bars + 7, *u_ready = bars + 8, *s_full = bars + 9,
           *o_full = bars + 10;
  uint64_t *o_read = bars + 11, *g_full = bars + 12, *g_empty = bars + 13;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + L::NUM_BARS);
  volatile uint32_t* abort_word = tmem_holder + 1;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1 + DK_CHAIN + DK_OUT);
    }
    mbar_init(s_ready, DK_CHAIN * 32);
    mbar_init(d1_full, 1);
    mbar_init(r_ready, DK_CHAIN * 32);
    mbar_init(d2_full, 1);
    mbar_init(u_ready, DK_CHAIN * 32);
    mbar_init(s_full, 1);
    mbar_init(o_full, 1);
    mbar_init(o_read, DK_OUT * 32);
    mbar_init(g_full, 1);
    mbar_init(g_empty, DK_OUT);
    *abort_word = 0;
    fence_barrier_init();
    prefetch_tensormap(&tm);
  }
  if (warp == DK_CHAIN + DK_OUT + 1) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  for (int i = tid; i < DC * 8; i += DK_THREADS) {
    const int r = i >> 3, c8 = i & 7;
    uint32_t w[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) w[j] = c8 * 8 + 2 * j == r ? 0x3f80u : (c8 * 8 + 2 * j + 1 == r ? 0x3f800000u : 0u);
    *reinterpret_cast<uint4*>(smem + L::OFF_ONE + dl_swz(r, c8)) = make_uint4(w[0], w[1], w[2], w[3]);
  }
  fence_proxy_async_smem();
  pdl_sync();
  const int seq = blockIdx.x / p.heads, h = blockIdx.x - seq * p.heads, hk = h / (p.heads / p.kv_heads), D = p.dim, E = p.vdim;
  const int row0 = p.cu[seq], rows = p.cu[seq + 1] - row0, slot = p.state_slots[seq];
  const bool live = slot >= 0 && slot < p.num_slots;
  if (slot >= p.num_slots && tid == 0) report_bad_arg(p.status, 52);
  const int chunks = live ? (rows + DC - 1) / DC : 0, chunk0 = p.chunk_cu[seq];
  const bool carried = rows > 0 && p.positions[row0] > 0;
  float* state = p.state + ((long long)(live ? slot : 0) * p.heads + h) * D * E;
  __nv_bfloat16* gy = reinterpret_cast<__nv_bfloat16*>(p.y) + (long long)row0 * p.ld_y + h * E;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;
  // columns: [S^T K^T, later U, later P U | S^T Q^T] 0 - 127, S^T 128 - 255, its parts 256 - 383, V^T, then R's, then U's parts 384 - 447, W's 448 - 511.
  // Parts lie as a warp stores them: the hi, then the lo halves of 16 columns (tokens or dims), one k-step of a product.
  const uint32_t T_D = tmem, T_S = tmem + 128, T_SP = tmem + 256, T_R = tmem + 384, T_W = tmem + 448;
  const int ksteps = (D + 15) / 16;
  bool ok = true;

  if (warp == DK_CHAIN + DK_OUT) {
    if (chunks > 0 && elect_one()) {
      const int pd = (D + 63) / 64, pe = (E + 63) / 64;
      for (int ch = 0; ch < chunks; ++ch) {
        const int st = ch & 1, at = row0 + ch * DC;
        if (!mbar_wait(&empty[st], ((ch >> 1) & 1) ^ 1, abort_word)) {
          *abort_word = ERR_WAIT_EMPTY;
          break;
        }
        uint8_t* s = smem + st * L::STAGE;
        mbar_expect_tx(&full[st], (uint32_t)(2 * pd + pe) * DC_TILE + DI_BYTES);
        for (int i = 0; i < pd; ++i) {
          tma_load_2d(s + i * 16384, &tm, &full[st], (p.kv_heads + hk) * D + i * 64, at);
          tma_load_2d(s + i * 16384 + DC_TILE, &tm, &full[st], hk * D + i * 64, at);
        }
        for (int i = 0; i < pe; ++i) tma_load_2d(s + L::X + i * DC_TILE, &tm, &full[st], 2 * p.kv_heads * D + h * E + i * 64, at);
        bulk_load(s + L::X + L::V, reinterpret_cast<const uint8_t*>(p.image) + ((long long)(chunk0 + ch) * p.heads + h) * DI_BYTES, DI_BYTES,
                  &full[st]);
      }
    }
  } else if (warp == DK_CHAIN + DK_OUT + 1) {
    if (chunks > 0 && elect_one()) {
      constexpr uint32_t id_x = make_idesc_bf16(128, 128, false, false), id_t = make_idesc_bf16(128, DC, false, false);
      constexpr uint32_t id_v = make_idesc_bf16(128, DC, true, false);
      const uint64_t one = make_smem_desc(smem_u32(smem + L::OFF_ONE), 16, 1024);
      const uint32_t id_k = make_idesc_bf16(128, ksteps * 16, false, true);
      for (int ch = 0; ch < chunks; ++ch) {
        const int st = ch & 1;
        const uint32_t ph = ch & 1;
        const uint32_t at = smem_u32(smem + st * L::STAGE), im = at + L::X + L::V;
        const uint64_t x = make_smem_desc(at, 16, 1024), kt = make_smem_desc(at, 16384, 1024);
        const uint64_t th = make_smem_desc(im + DI_T, 16, 1024), tl = make_smem_desc(im + DI_T + DC_TILE, 16, 1024);
        const uint64_t ph_ = make_smem_desc(im + DI_P, 16, 1024), pl = make_smem_desc(im + DI_P + DC_TILE, 16, 1024);
        const uint64_t vt = make_smem_desc(at + L::X, DC_TILE, 1024);
        ok = mbar_wait(&full[st], (ch >> 1) & 1, abort_word);
        if (!ok) break;
#pragma unroll
        for (int k = 0; k < 4; ++k) umma_f16_ss(T_R, vt + (uint32_t)(k * 128), one + (uint32_t)(k * 2), id_v, k ? 1u : 0u);
        ok = mbar_wait(s_ready, ph, abort_word) && (ch == 0 || mbar_wait(o_read, ph ^ 1, abort_word));
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int part = 0; part < 2; ++part)
          for (int k = 0; k < ksteps; ++k)
            umma_f16_ts(T_D, T_SP + k * 16 + part * 8, x + (uint32_t)(((k / 4) * 16384 + (k % 4) * 32) >> 4), id_x, (part | k) ? 1u : 0u);
        umma_commit(d1_full);
        ok = mbar_wait(r_ready, ph, abort_word);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int part = 0; part < 3; ++part)         // hi hi, hi lo, lo hi
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_f16_ts(T_D, T_R + k * 16 + (part == 2 ? 8 : 0), (part == 1 ? tl : th) + (uint32_t)(k * 2), id_t, (part | k) ? 1u : 0u);
        umma_commit(d2_full);
        ok = mbar_wait(u_ready, ph, abort_word);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16_ts(T_S, T_W + k * 16 + part * 8, kt + (uint32_t)(k * 128), id_k, 1u);
        umma_commit(s_full);
#pragma unroll
        for (int part = 0; part < 3; ++part)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_f16_ts(T_D, T_R + k * 16 + (part == 2 ? 8 : 0), (part == 1 ? pl : ph_) + (uint32_t)(k * 2), id_t, (part | k) ? 1u : 0u);
        umma_commit(o_full);
        umma_commit(&empty[st]);
      }
      if (!ok) *abort_word = ERR_WAIT_TMEM_FULL;
    }
  } else if (warp < DK_CHAIN) {
    const int quarter = warp & 3, cg = warp >> 2, e = quarter * 32 + lane;        // this thread's column of v; half of the tokens or dims
    const uint32_t la = uint32_t(quarter * 32) << 16;
    constexpr int HD = PD * 64 / (DK_CHAIN / 4), HT = DC / (DK_CHAIN / 4);        // dims of S and tokens a thread looks after
    // 16 dims of S: the parts into operand places, times the chunk's decay into the accumulator
    auto publish = [&](uint32_t (&raw)[16], int d0, float g) __attribute__((always_inline)) {
      uint32_t parts[16];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (d0 + 2 * i >= D) raw[2 * i] = raw[2 * i + 1] = 0u;       // dim is even
        dl_split2(__uint_as_float(raw[2 * i]), __uint_as_float(raw[2 * i + 1]), parts[i], parts[8 + i]);
      }
      tmem_st_32x16(T_SP + la + d0, parts);
#pragma unroll
      for (int i = 0; i < 16; ++i) raw[i] = __float_as_uint(__uint_as_float(raw[i]) * g);
      tmem_st_32x16(T_S + la + d0, raw);
    };
    auto signal = [&](uint64_t* bar) {
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(bar);
    };
    // One warp polls, the others sleep at the barrier behind it and leave the issue slots to the output warps.
    // After a wait that gave up the loop goes on, without waiting, so that the warps meet at every barrier.
    auto wait = [&](uint64_t* bar, uint32_t parity) {
      if (warp == 0 && !mbar_wait(bar, parity, abort_word)) *abort_word = ERR_WAIT_MISC;
      __syncwarp();
      asm volatile("bar.sync 3, %0;" ::"n"(DK_CHAIN * 32) : "memory");
      tc_fence_after();
    };
    if (chunks > 0) {
      wait(&full[0], 0);
      const float g = reinterpret_cast<const float*>(smem + L::X + L::V + DI_F)[4 * DC];
#pragma unroll 1
      for (int d0 = cg * HD; d0 < (cg + 1) * HD; d0 += 16) {
        uint32_t raw[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) raw[i] = carried && e < E && d0 + i < D ? __float_as_uint(state[(long long)(d0 + i) * E + e]) : 0u;
        publish(raw, d0, g);
      }
      signal(s_ready);
    }
    for (int ch = 0; ch < chunks; ++ch) {
      const int st = ch & 1;
      const uint32_t ph = ch & 1;
      const uint8_t* stage = smem + st * L::STAGE;
      const float* f = reinterpret_cast<const float*>(stage + L::X + L::V + DI_F) + cg * HT;
      uint32_t parts[16], d[16];                     // (the stage has landed: its decay was read a chunk ago)
      wait(d1_full, ph);
#pragma unroll
      for (int q = 0; q < HT / 16; ++q) {
        uint32_t v[16];
        tmem_ld_32x16(T_D + la + cg * HT + q * 16, d);
        tmem_ld_32x16(T_R + la + cg * HT + q * 16, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float4 w = *reinterpret_cast<const float4*>(f + cg * HT + q * 32 + 4 * i);
          const float x = e < E ? __uint_as_float(v[2 * i]) : 0.f, y = e < E ? __uint_as_float(v[2 * i + 1]) : 0.f;
          dl_split2(fmaf(w.y, __uint_as_float(d[2 * i]), w.x * x), fmaf(w.w, __uint_as_float(d[2 * i + 1]), w.z * y), parts[i], parts[8 + i]);
        }
        tmem_st_32x16(T_R + la + cg * HT + q * 16, parts);
      }
      signal(r_ready);
      wait(d2_full, ph);
#pragma unroll
      for (int q = 0; q < HT / 16; ++q) {
        tmem_ld_32x16(T_D + la + cg * HT + q * 16, d);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float2 w = *reinterpret_cast<const float2*>(f + 2 * DC + q * 16 + 2 * i);
          dl_split2(__uint_as_float(d[2 * i]) * w.x, __uint_as_float(d[2 * i + 1]) * w.y, parts[i], parts[8 + i]);
        }
        tmem_st_32x16(T_W + la + cg * HT + q * 16, parts);
#pragma unroll
        for (int i = 0; i < 8; ++i) dl_split2(__uint_as_float(d[2 * i]), __uint_as_float(d[2 * i + 1]), parts[i], parts[8 + i]);
        tmem_st_32x16(T_R + la + cg * HT + q * 16, parts);
      }
      signal(u_ready);
      __syncwarp();
      if (lane == 0) mbar_arrive(&empty[st]);        // nothing of the stage is read here any more
      if (ch + 1 == chunks) break;
      wait(&full[st ^ 1], ((ch + 1) >> 1) & 1);
      const float g = reinterpret_cast<const float*>(smem + (st ^ 1) * L::STAGE + L::X + L::V + DI_F)[4 * DC];
      wait(s_full, ph);
#pragma unroll
      for (int piece = 0; piece < HD / 16; ++piece) {
        const int d0 = cg * HD + piece * 16;
        tmem_ld_32x16(T_S + la + d0, d);
        tmem_ld_wait();
        publish(d, d0, g);
      }
      signal(s_ready);
    }
    if (chunks > 0) {
      wait(s_full, (chunks - 1) & 1);
#pragma unroll 1
      for (int d0 = cg * HD; d0 < (cg + 1) * HD; d0 += 16) {
        uint32_t raw[16];
        tmem_ld_32x16(T_S + la + d0, raw);
        tmem_ld_wait();
        if (e < E && *abort_word == 0) {
#pragma unroll
          for (int i = 0; i < 16; ++i)
            if (d0 + i < D) state[(long long)(d0 + i) * E + e] = __uint_as_float(raw[i]);
        }
      }
    }
  } else {
    const int quarter = warp & 3, e = quarter * 32 + lane, ow = warp - DK_CHAIN, og = ow >> 2;       // half of the tokens
    const uint32_t la = uint32_t(quarter * 32) << 16;
    float* o = reinterpret_cast<float*>(smem + L::OFF_O);
    constexpr int OP = PE * 64, HT = DC / (DK_OUT / 4), RT = DC / DK_OUT;       // tokens read from tensor memory, and finished, per warp
    const int c = lane * 4;                          // columns of an output row that this lane finishes
    float w[4] = {0.f, 0.f, 0.f, 0.f};
    if (c < E) load_vec<4>(reinterpret_cast<const __nv_bfloat16*>(p.weight) + c, w);
    const float share = 1.f / (float)E;
    const uint8_t* gate = smem + L::OFF_G + (c < E ? (c >> 6) * DC_TILE + (c & 7) * 2 : 0);
    auto load_gates = [&](int ch) {                  // by one thread, once the gates of the chunk before have been used
      mbar_expect_tx(g_full, (uint32_t)((E + 63) / 64) * DC_TILE);
      for (int i = 0; i < (E + 63) / 64; ++i) tma_load_2d(smem + L::OFF_G + i * DC_TILE, &tm_gate, g_full, h * E + i * 64, row0 + ch * DC);
    };
    if (chunks > 0 && warp == DK_CHAIN && lane == 0) load_gates(0);
    __syncwarp();
    for (int ch = 0; ch < chunks; ++ch) {
      const int st = ch & 1, n = min(DC, rows - ch * DC);
      const float* f = reinterpret_cast<const float*>(smem + st * L::STAGE + L::X + L::V + DI_F) + 3 * DC + og * HT;
      if (warp == DK_CHAIN && (!mbar_wait(&full[st], (ch >> 1) & 1, abort_word) || !mbar_wait(g_full, ch & 1, abort_word) ||
                               !mbar_wait(o_full, ch & 1, abort_word)))
        *abort_word = ERR_WAIT_TMEM_FULL;
      __syncwarp();
      asm volatile("bar.sync 2, %0;" ::"n"(DK_OUT * 32) : "memory");      // the rows of the chunk before have been read, too
      tc_fence_after();
      float r[HT];
#pragma unroll
      for (int q = 0; q < HT / 16; ++q) {
        uint32_t a[16], b[16];
        tmem_ld_32x16(T_D + la + 64 + og * HT + q * 16, a);
        tmem_ld_32x16(T_D + la + og * HT + q * 16, b);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) r[q * 16 + i] = fmaf(f[q * 16 + i], __uint_as_float(a[i]), __uint_as_float(b[i]));
      }
      tc_fence_before();
      mbar_arrive(o_read);
      __syncwarp();
      if (lane == 0) mbar_arrive(&empty[st]);
      if (e < OP) {
#pragma unroll
        for (int i = 0; i < HT; ++i) o[(og * HT + i) * OP + e] = r[i];
      }
      asm volatile("bar.sync 2, %0;" ::"n"(DK_OUT * 32) : "memory");
      // rows ow, ow + DK_OUT, ... of the chunk, all of them at a time
      float x[RT][4], ss[RT], g[4];
#pragma unroll
      for (int j = 0; j < RT; ++j) {
#pragma unroll
        for (int i = 0; i < 4; ++i) x[j][i] = 0.f;
        if (c < E) load_vec<4>(o + (ow + j * DK_OUT) * OP + c, x[j]);
        ss[j] = fmaf(x[j][0], x[j][0], fmaf(x[j][1], x[j][1], fmaf(x[j][2], x[j][2], x[j][3] * x[j][3])));
      }
#pragma unroll
      for (int k = 16; k > 0; k >>= 1)
#pragma unroll
        for (int j = 0; j < RT; ++j) ss[j] += __shfl_xor_sync(0xffffffffu, ss[j], k);
      __nv_bfloat16* yr = gy + (long long)(ch * DC + ow) * p.ld_y + c;
#pragma unroll
      for (int j = 0; j < RT; ++j) {
        const int t = ow + j * DK_OUT;
        const float inv = rsqrtf(fmaf(ss[j], share, p.eps));
        load_vec<4>(reinterpret_cast<const __nv_bfloat16*>(gate + dl_swz(t, (c >> 3) & 7)), g);
#pragma unroll
        for (int i = 0; i < 4; ++i) x[j][i] *= inv * w[i] * g[i] * dl_sigmoid(g[i]);
        if (t < n && c < E) store_vec<4>(yr, x[j]);
        yr += DK_OUT * p.ld_y;
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(g_empty);
      if (warp == DK_CHAIN && lane == 0 && ch + 1 < chunks) {
        if (mbar_wait(g_empty, ch & 1, abort_word)) load_gates(ch + 1);
        else *abort_word = ERR_WAIT_EMPTY;
      }
      __syncwarp();
    }
  }
  if (!live) {
    for (int t = warp; t < rows; t += DK_THREADS / 32)
      for (int c = lane * 8; c < E; c += 256) *reinterpret_cast<uint4*>(gy + (long long)t * p.ld_y + c) = make_uint4(0, 0, 0, 0);
  }
  __syncwarp();
  tc_fence_before();
  __syncthreads();
  if (*abort_word != 0) {
    if (tid == 0 && p.status != nullptr) atomicCAS(p.status, 0u, (*abort_word) | (blockIdx.x << 8));
    const uint64_t w0 = globaltimer_ns();
    while (globaltimer_ns() - w0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == DK_CHAIN + DK_OUT + 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

template <int PD, int PE>
static int launch_delta_chunk(const CUtensorMap& tm, const CUtensorMap& tm_gate, const DeltaArgs& p, cudaStream_t st) {
  auto kern = delta_chunk_kernel<PD, PE>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, DeltaChunkSmem<PD, PE>::TOTAL) != cudaSuccess ||
        cudaFuncSetAttribute(delta_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, DeltaPrepareSmem::TOTAL) != cudaSuccess)
      return -3;
    configured = true;
  }
  const int sets = (p.heads / p.kv_heads + DP_HEADS - 1) / DP_HEADS;
  launch_dep(delta_prepare_kernel, (unsigned)(p.chunks * p.kv_heads * sets), 128, DeltaPrepareSmem::TOTAL, st, tm, p);
  launch_dep(kern, (unsigned)(p.seqs * p.heads), DK_THREADS, DeltaChunkSmem<PD, PE>::TOTAL, st, tm, tm_gate, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <typename T>
static int launch_delta(const DeltaArgs& p, bool vec, bool step, size_t smem, int rows_per_thread, cudaStream_t st) {
  if (step) {
    const unsigned blocks = (unsigned)((long long)p.seqs * p.heads);
    if (rows_per_thread <= 4) launch_dep(delta_step_kernel<T, 4>, blocks, 256, smem, st, p);
    else launch_dep(delta_step_kernel<T, 16>, blocks, 256, smem, st, p);
  } else {
    const dim3 grid(p.seqs, p.heads);
    if (vec) launch_dep(delta_recurrent_kernel<T, 4>, grid, 256, smem, st, p);
    else launch_dep(delta_recurrent_kernel<T, 1>, grid, 256, smem, st, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_delta_image_bytes(void) { return DI_BYTES; }
extern "C" int b200_delta_chunk_tokens(void) { return DC; }

// See DeltaArgs.  mode 0: one row per sequence or rows in order; 1: chunked (bf16, cu and ab given, dim and vdim multiples of 8 up to 128).
extern "C" int b200_delta(const DeltaArgs* args, int mode, int f32, cudaStream_t st) {
  const DeltaArgs& p = *args;
  if (p.seqs <= 0 || p.rows <= 0) return 0;
  if (p.heads <= 0 || p.kv_heads <= 0 || p.heads % p.kv_heads || p.heads > 65535 || p.dim <= 0 || p.vdim <= 0 || p.num_slots <= 0) return -10;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(p.c) | reinterpret_cast<uintptr_t>(p.state);
  if (mode == 1) {
    if (f32 || p.cu == nullptr || p.chunk_cu == nullptr || p.ab == nullptr || p.image == nullptr || p.taps > 0 || p.dim > 128 || p.vdim > 128 ||
        p.dim % 8 || p.vdim % 8 || p.chunks <= 0)
      return -11;
    if (p.ld_c % 8 || p.ld_y % 8 || p.ld_gate % 8 ||
        ((ptrs | reinterpret_cast<uintptr_t>(p.y) | reinterpret_cast<uintptr_t>(p.image) | reinterpret_cast<uintptr_t>(p.weight)) & 15) ||
        (reinterpret_cast<uintptr_t>(p.gate) & 15))
      return -11;
    CUtensorMap tm, tm_gate;
    if (make_tmap_bf16_2d(&tm_gate, p.gate, (uint64_t)p.rows, (uint64_t)p.heads * p.vdim, (uint64_t)p.ld_gate, 64, DC)) return -20;
    if (make_tmap_bf16_2d(&tm, p.c, (uint64_t)p.rows, (uint64_t)(2 * p.kv_heads * p.dim + p.heads * p.vdim), (uint64_t)p.ld_c, 64, DC)) return -20;
    if (p.dim <= 64) return p.vdim <= 64 ? launch_delta_chunk<1, 1>(tm, tm_gate, p, st) : launch_delta_chunk<1, 2>(tm, tm_gate, p, st);
    return p.vdim <= 64 ? launch_delta_chunk<2, 1>(tm, tm_gate, p, st) : launch_delta_chunk<2, 2>(tm, tm_gate, p, st);
  }
  const bool vec = p.vdim % 4 == 0 && p.ld_c % 4 == 0 && (ptrs & 15) == 0;
  const int groups = vec ? p.vdim / 4 : p.vdim, rg = groups < 256 ? 256 / groups : 1, per = (p.dim + rg - 1) / rg;
  const size_t smem = ((size_t)(2 * p.dim + 2 * p.vdim + 3) / 4 * 4 + 2ull * rg * p.vdim) * sizeof(float);
  if (smem > 48 * 1024) return -12;
  const bool step = vec && p.cu == nullptr && groups <= 256 && per <= 16;
  if ((p.ab == nullptr || p.taps > 0) && !step) return -13;
  if (p.ab == nullptr && (p.h == nullptr || p.w_ab == nullptr || p.width <= 0 || p.ld_h % 4 || p.ld_w % 4 ||
                          ((reinterpret_cast<uintptr_t>(p.h) | reinterpret_cast<uintptr_t>(p.w_ab)) & 15)))
    return -13;
  if (p.taps > 0 && (p.filter == nullptr || p.ring == nullptr)) return -13;
  return f32 ? launch_delta<float>(p, vec, step, smem, per, st) : launch_delta<__nv_bfloat16>(p, vec, step, smem, per, st);
}
