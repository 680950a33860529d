// Matrix memory with exponential gates (mLSTM of xLSTM).  Per head, with log gates i_t (input) and f_t (forget), both capped softly,
//     m_t = max(f_t + m_(t-1), i_t)                        running maximum, m_0 = 0
//     S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,    n_t likewise with k_t alone
//     o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
// then o_t / rms(o_t) * weight * sigmoid(gate).  q carries dim^(-1/2).  A request's state of a head is fp32 and contiguous:
// S (dim, vdim) | n (dim) | m, rounded up to 4 floats; it lives in a slot.  The gates' projections arrive in fp32.
#include "typed.cuh"

namespace b200 {

int make_tmap_bf16_2d(CUtensorMap* tm, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_cols,
                      uint32_t box_rows);

struct MlstmParams {
  const void* proj;          // (rows, ld_proj): q | k | v | gate, heads contiguous inside each
  long long ld_proj;
  const float* gates;        // (rows, ld_gates): input gate pre-activations of all heads | forget gates; null: the decode step
  long long ld_gates;        // takes the products of its input row with the gates' weights itself
  const void *h, *w_gates;   // gates null: (rows, ld_h) and (2 * heads, ld_wg), `width` columns
  long long ld_h, ld_wg;
  int width;
  const float* gate_bias;    // (2 * heads), the same order
  const void* weight;        // (heads * vdim)
  void* y;                   // (rows, ld_y)
  long long ld_y;
  float* state;              // (slots, heads, stride)
  const int* state_slots;    // per sequence of the launch; negative = padding
  const int* cu;             // optional (seqs + 1): rows of each sequence; null = one row per sequence
  const int* positions;      // per row of the launch
  int seqs, rows, heads, dim, vdim, stride, num_slots;
  float cap, eps;
  uint32_t* status;
};

__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) {
  const float s = cap * tanhf(z / cap);
  return fminf(s, 0.f) - log1pf(expf(-fabsf(s)));
}

// One block per (sequence, head), tokens in order, the state in global memory (every thread re-reads only what it wrote): any
// dim and vdim, T = bf16 or fp32.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) mlstm_recurrent_kernel(const MlstmParams p) {
  pdl_sync();
  extern __shared__ float msm[];
  __shared__ float red[32];
  const int seq = blockIdx.x, h = blockIdx.y;
  const int D = p.dim, E = p.vdim;
  const int groups = E / VEC, cgt = groups < 256 ? groups : 256, rg = 256 / cgt;
  float *qs = msm, *ks = msm + D, *part = msm + 2 * D;          // [D], [D], [rg][E]
  const int ty = threadIdx.x / cgt, tx = threadIdx.x - ty * cgt;
  const int row0 = p.cu != nullptr ? p.cu[seq] : seq, row1 = p.cu != nullptr ? p.cu[seq + 1] : seq + 1;
  const int slot = p.state_slots[seq];
  const T* proj = reinterpret_cast<const T*>(p.proj);
  T* y = reinterpret_cast<T*>(p.y);
  if (slot < 0 || slot >= p.num_slots) {
    if (slot >= p.num_slots && threadIdx.x == 0) report_bad_arg(p.status, 17);
    for (int row = row0; row < row1; ++row)
      for (int c = threadIdx.x; c < E; c += 256) from_f(y[(long long)row * p.ld_y + h * E + c], 0.f);
    return;
  }
  float* S = p.state + ((long long)slot * p.heads + h) * p.stride;
  float* N = S + (long long)D * E;
  const float qscale = rsqrtf((float)D);
  const float bi = p.gate_bias[h], bf = p.gate_bias[p.heads + h];
  float m = 0.f;
  for (int row = row0; row < row1; ++row) {
    const bool fresh = p.positions[row] == 0;        // a sequence starts from the zero state, whatever its slot held
    if (fresh) m = 0.f;
    else if (row == row0) m = N[D];
    const T* pr = proj + (long long)row * p.ld_proj;
    const T *qr = pr + h * D, *kr = pr + p.heads * D + h * D, *vr = pr + 2 * p.heads * D + h * E;
    const T* gr = pr + 2 * p.heads * D + p.heads * E + h * E;
    const float* gt = p.gates + (long long)row * p.ld_gates;
    const float li = log_input_gate(gt[h] + bi, p.cap), lf = log_forget_gate(gt[p.heads + h] + bf, p.cap);
    const float mn = fmaxf(lf + m, li), keep = expf(lf + m - mn), take = expf(li - mn);
    m = mn;
    float den = 0.f;
    for (int d = threadIdx.x; d < D; d += 256) {
      const float qv = to_f(qr[d]) * qscale, kv = to_f(kr[d]) * take;
      qs[d] = qv;
      ks[d] = kv;
      const float nv = fresh ? kv : fmaf(keep, N[d], kv);
      N[d] = nv;
      den = fmaf(nv, qv, den);
    }
    den = block_total(den, red);                     // its barriers also publish qs and ks
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
            s[i] = fmaf(keep, s[i], kd * v[i]);
            o[i] = fmaf(s[i], qd, o[i]);
          }
          store_vec<VEC>(sp, s);
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) part[ty * E + g * VEC + i] = o[i];
      }
    }
    __syncthreads();
    const float low = 1.f / (fmaxf(fabsf(den), expf(-m)) + 1e-6f);
    float ss = 0.f;
    for (int c = threadIdx.x; c < E; c += 256) {
      float o = 0.f;
      for (int r = 0; r < rg; ++r) o += part[r * E + c];
      o *= low;
      part[c] = o;                                   // row 0 of this column is read by this thread only
      ss += o * o;
    }
    const float inv = rsqrtf(block_total(ss, red) / (float)E + p.eps);
    const T* wr = reinterpret_cast<const T*>(p.weight) + h * E;
    for (int c = threadIdx.x; c < E; c += 256)
      from_f(y[(long long)row * p.ld_y + h * E + c], part[c] * inv * to_f(wr[c]) / (1.f + expf(-to_f(gr[c]))));
    __syncthreads();
  }
  if (threadIdx.x == 0 && row1 > row0) N[D] = m;
}

// Decode step of a state that fits the block's registers (NR rows of four columns per thread): one block per (request, head); the
// whole state is requested before anything else, so the gates and the small products run under its latency.
template <typename T, int NR>
__global__ void __launch_bounds__(256, NR > 8 ? 2 : 3) mlstm_step_kernel(const MlstmParams p) {
  pdl_sync();
  extern __shared__ float msm[];
  __shared__ float red[32];
  const int seq = blockIdx.x / p.heads, h = blockIdx.x - seq * p.heads;
  const int D = p.dim, E = p.vdim, groups = E / 4, rg = 256 / groups;
  float *qs = msm, *ks = msm + D, *part = msm + 2 * D;         // [D], [D], [rg][E]
  const int ty = threadIdx.x / groups, tx = threadIdx.x - ty * groups;
  const int slot = p.state_slots[seq];
  const T* pr = reinterpret_cast<const T*>(p.proj) + (long long)seq * p.ld_proj;
  T* y = reinterpret_cast<T*>(p.y) + (long long)seq * p.ld_y + h * E;
  if (slot < 0 || slot >= p.num_slots) {
    if (slot >= p.num_slots && threadIdx.x == 0) report_bad_arg(p.status, 17);
    for (int c = threadIdx.x; c < E; c += 256) from_f(y[c], 0.f);
    return;
  }
  const bool fresh = p.positions[seq] == 0, on = ty < rg;
  float* base = p.state + ((long long)slot * p.heads + h) * p.stride;
  float* N = base + (long long)D * E;
  float4* S = reinterpret_cast<float4*>(base) + tx;
  // the gates' operands are few and in L2: the first of them are requested before the state, not behind it
  float hx[4] = {0.f, 0.f, 0.f, 0.f}, hi[4] = {0.f, 0.f, 0.f, 0.f}, hf[4] = {0.f, 0.f, 0.f, 0.f};
  const T* hr = reinterpret_cast<const T*>(p.h) + (long long)seq * p.ld_h;
  const T* wi = reinterpret_cast<const T*>(p.w_gates) + (long long)h * p.ld_wg;
  const T* wf = wi + (long long)p.heads * p.ld_wg;
  if (p.gates == nullptr && threadIdx.x * 4 < p.width) {
    load_vec<4>(hr + threadIdx.x * 4, hx);
    load_vec<4>(wi + threadIdx.x * 4, hi);
    load_vec<4>(wf + threadIdx.x * 4, hf);
  }
  float4 s[NR];
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = ty + j * rg;
    s[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on && d < D && !fresh) s[j] = __ldcs(S + (long long)d * groups);
  }
  const float m = fresh ? 0.f : N[D];
  float zi = 0.f, zf = 0.f;
  if (p.gates != nullptr) {
    const float* gt = p.gates + (long long)seq * p.ld_gates;
    zi = gt[h];
    zf = gt[p.heads + h];
  } else {
    for (int c = threadIdx.x * 4; c < p.width; c += 1024) {            // pitches are multiples of 4, what lies in the pads is left out
      if (c >= 1024) {
        load_vec<4>(hr + c, hx);
        load_vec<4>(wi + c, hi);
        load_vec<4>(wf + c, hf);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float xv = c + i < p.width ? hx[i] : 0.f;
        zi = fmaf(xv, hi[i], zi);
        zf = fmaf(xv, hf[i], zf);
      }
    }
    zi = block_total(zi, red);
    zf = block_total(zf, red);
  }
  const float li = log_input_gate(zi + p.gate_bias[h], p.cap);
  const float lf = log_forget_gate(zf + p.gate_bias[p.heads + h], p.cap);
  const float mn = fmaxf(lf + m, li), keep = expf(lf + m - mn), take = expf(li - mn);
  const float qscale = rsqrtf((float)D);
  const T *qr = pr + h * D, *kr = pr + p.heads * D + h * D;
  float den = 0.f;
  for (int d = threadIdx.x; d < D; d += 256) {
    const float qv = to_f(qr[d]) * qscale, kv = to_f(kr[d]) * take;
    qs[d] = qv;
    ks[d] = kv;
    const float nv = fresh ? kv : fmaf(keep, N[d], kv);
    N[d] = nv;
    den = fmaf(nv, qv, den);
  }
  float v[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) load_vec<4>(pr + 2 * p.heads * D + h * E + tx * 4, v);
  den = block_total(den, red);                       // its barriers also publish qs and ks, and m has been read
  if (threadIdx.x == 0) N[D] = mn;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = ty + j * rg;
    if (!on || d >= D) continue;
    const float kd = ks[d], qd = qs[d];
    s[j].x = fmaf(keep, s[j].x, kd * v[0]); s[j].y = fmaf(keep, s[j].y, kd * v[1]);
    s[j].z = fmaf(keep, s[j].z, kd * v[2]); s[j].w = fmaf(keep, s[j].w, kd * v[3]);
    o.x = fmaf(s[j].x, qd, o.x); o.y = fmaf(s[j].y, qd, o.y); o.z = fmaf(s[j].z, qd, o.z); o.w = fmaf(s[j].w, qd, o.w);
    __stcs(S + (long long)d * groups, s[j]);
  }
  if (on) *reinterpret_cast<float4*>(part + ty * E + tx * 4) = o;
  __syncthreads();
  const float low = 1.f / (fmaxf(fabsf(den), expf(-mn)) + 1e-6f);
  float ss = 0.f, mine[4];
  int n = 0;
  for (int c = threadIdx.x; c < E && n < 4; c += 256, ++n) {           // E <= 1024
    float t = 0.f;
    for (int r = 0; r < rg; ++r) t += part[r * E + c];
    mine[n] = t * low;
    ss += mine[n] * mine[n];
  }
  const float inv = rsqrtf(block_total(ss, red) / (float)E + p.eps);
  const T* gr = pr + 2 * p.heads * D + p.heads * E + h * E;
  const T* wr = reinterpret_cast<const T*>(p.weight) + h * E;
  n = 0;
  for (int c = threadIdx.x; c < E && n < 4; c += 256, ++n)
    from_f(y[c], mine[n] * inv * to_f(wr[c]) * sigmoid_f(to_f(gr[c])));
}

// ------------------------------------------------------------------------------------ prompts, bf16, on the tensor cores
// One CTA = one (portion, head), chunks of n <= 128 tokens in order.  Inside a chunk let F_t = f_1 + ... + f_t, a_s = i_s - F_s and
// M_t = max(m_prev, a_1 .. a_t), so that m_t = F_t + M_t.  Then
//     S_t^T q_t = exp(m_prev - M_t) S_prev^T q_t + sum_(s <= t) exp(a_s - M_t) (q_t . k_s) v_s
// and S_next = exp(m_prev - M_n) S_prev + sum_s exp(a_s - M_n) k_s v_s^T; every exponent is at most zero.  As products:
//     scores = Q K^T    O_inter = Q S_prev    P = scores * exp(a_s - M_t), causal    O_intra = P V    S_next = g S_prev + K~^T V
// q, k, v are bf16 as projected and enter unrounded; what the gates or the state make fp32 (P, K~, S_prev) is split into two
// bf16 parts (hi + lo, 16 significant bits) whose products accumulate in fp32.  n . q is kept beside it on the FMA pipes.
//   tensor memory: scores, then P [0, 128)  O_inter [128, 128 + EP)  O_intra [256, 256 + EP)  S [384, 384 + EP)
//   shared memory: Q | K, then K~ hi | K~ lo, later the outputs on their way | V | S_prev hi, lo, all 128-byte swizzled panels
// Sixteen warps do the element-wise phases (four warps per 32 lanes of tensor memory, a quarter of the columns each); one of them,
// which has no score that is not masked, also issues TMA and MMAs and scans the next chunk's gates.  The output gates come in and
// the outputs go out through K~ lo's place, in whole rows.
constexpr int ML_CHUNK = 128;
constexpr int ML_THREADS = 512;
constexpr int ML_ISSUER = 12;             // rows 0 - 31, keys 96 - 127
constexpr float ML_NEVER = -1e30f;        // log input gate of a token that is not there

template <int EP>
struct MlstmSmem {
  static constexpr int TILE = 32768;                 // 128 rows x 128 columns of bf16: two panels
  static constexpr int VT = EP / 64 * 16384;
  static constexpr int OFF_Q = 0, OFF_K = TILE, OFF_KL = 2 * TILE, OFF_V = 3 * TILE;
  static constexpr int OFF_SH = OFF_V + VT, OFF_SL = OFF_SH + VT, OFF_F = OFF_SL + VT;
  // floats: a, M [2][128] in log2 units, m_t [2][128]; n [128]; den, sum of squares [4][128] each; column sums of K~ [4096];
  // the heads' weight [128]; m_prev [2]
  static constexpr int FLOATS = 3 * 256 + 128 + 2 * 512 + 4096 + 128 + 4;
  static constexpr int OFF_BAR = OFF_F + FLOATS * 4;
  static constexpr int TOTAL = OFF_BAR + 5 * 8 + 16 + 1024;
};

// 16-byte piece `c8` (8 columns) of row `r` in a tile of 64-column panels, 128-byte swizzle
__device__ __forceinline__ uint32_t ml_swz(int r, int c8) {
  return (uint32_t)(c8 >> 3) * 16384u + (uint32_t)r * 128u + (uint32_t)(((c8 & 7) ^ (r & 7)) << 4);
}
__device__ __forceinline__ void ml_unpack8(const uint4& v, float (&f)[8]) {
  const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y), c = unpack_bf16x2(v.z), d = unpack_bf16x2(v.w);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
}
// Two values as hi + lo, both bf16: hi is cut off (the remainder is exact), lo rounded.  Integer and FMA pipes only: the conversion
// unit shares its port with ex2.
__device__ __forceinline__ void ml_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const uint32_t a = __float_as_uint(x), b = __float_as_uint(y);
  hi = __byte_perm(a, b, 0x7632);
  lo = pack_bf16x2_alu(x - __uint_as_float(a & 0xffff0000u), y - __uint_as_float(b & 0xffff0000u));
}
__device__ __forceinline__ void ml_split8(const float (&x)[8], uint4& hi, uint4& lo) {
  ml_split2(x[0], x[1], hi.x, lo.x);
  ml_split2(x[2], x[3], hi.y, lo.y);
  ml_split2(x[4], x[5], hi.z, lo.z);
  ml_split2(x[6], x[7], hi.w, lo.w);
}
__device__ __forceinline__ float ml_exp2(float x) {       // x <= 0; far below zero gives zero
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float ml_sigmoid(float g) {    // (1 + tanh(g / 2)) / 2
  float t;
  asm("tanh.approx.f32 %0, %1;" : "=f"(t) : "f"(0.5f * g));
  return fmaf(0.5f, t, 0.5f);
}
template <int N>                                          // 16 or 32 columns of tensor memory
__device__ __forceinline__ void ml_tmem_ld(uint32_t addr, uint32_t (&r)[N]) {
  if constexpr (N == 32) tmem_ld_32x32(addr, r);
  else tmem_ld_32x16(addr, r);
}
template <int N>
__device__ __forceinline__ void ml_tmem_st(uint32_t addr, const uint32_t (&r)[N]) {
  if constexpr (N == 32) tmem_st_32x32(addr, r);
  else tmem_st_32x16(addr, r);
}

template <int EP>
__global__ void __launch_bounds__(ML_THREADS, 1) mlstm_chunk_kernel(const __grid_constant__ CUtensorMap tm_proj, const MlstmParams p) {
  using L = MlstmSmem<EP>;
  constexpr int HE = EP / 4;                          // columns of O and S that a thread handles
  constexpr float LOG2E = 1.4426950408889634f;
  extern __shared__ uint8_t ml_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ml_raw) + 1023) & ~uintptr_t(1023));
  float* sa = reinterpret_cast<float*>(smem + L::OFF_F);      // [2][128] a_s, log2 units
  float *sM = sa + 256, *sm = sM + 256, *sn = sm + 256;       // [2][128] M_t, log2 units; [2][128] m_t; [128] n
  float *sden = sn + 128, *srms = sden + 512, *scol = srms + 512, *sw = scol + 4096, *sprev = sw + 128;   // m_prev of chunk ch in sprev[ch & 1]
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR);
  uint64_t *bar_a = bars, *bar_s = bars + 1, *bar_o = bars + 2, *bar_l = bars + 3, *bar_g = bars + 4;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + 5);
  volatile uint32_t* abort_word = tmem_holder + 1;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bool issuer = warp == ML_ISSUER;

  if (tid == 0) {
    for (int i = 0; i < 5; ++i) mbar_init(&bars[i], 1);
    *abort_word = 0;
    fence_barrier_init();
    prefetch_tensormap(&tm_proj);
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  for (int i = tid; i < (L::OFF_F >> 4); i += ML_THREADS) reinterpret_cast<uint4*>(smem)[i] = make_uint4(0, 0, 0, 0);
  pdl_sync();
  const int seq = blockIdx.x / p.heads, h = blockIdx.x - seq * p.heads;
  const int D = p.dim, E = p.vdim;
  if (tid < 128) sw[tid] = tid < E ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.weight)[h * E + tid]) : 0.f;
  fence_proxy_async_smem();           // the zeros above come before what TMA writes
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;

  const int row0 = p.cu[seq], rows = p.cu[seq + 1] - row0;
  const int slot = p.state_slots[seq];
  const bool live = slot >= 0 && slot < p.num_slots;
  if (!live && slot >= p.num_slots && tid == 0) report_bad_arg(p.status, 18);
  const int pos0 = rows > 0 ? p.positions[row0] : 0;
  float* state = p.state + ((long long)(live ? slot : 0) * p.heads + h) * p.stride;
  float* state_n = state + (long long)D * E;
  const int quarter = warp & 3, cg = warp >> 2;       // lanes of tensor memory, group of columns
  const int r = quarter * 32 + lane;                  // this thread's row of tensor memory: a token, or a dim of S
  const int e0 = cg * HE;                             // its first column of O and S
  __nv_bfloat16* gy = reinterpret_cast<__nv_bfloat16*>(p.y) + (long long)row0 * p.ld_y + h * E;
  const float* gates = p.gates + (long long)row0 * p.ld_gates + h;
  const uint32_t lane_addr = uint32_t(quarter * 32) << 16;
  const uint32_t tm_a = tmem + lane_addr + cg * 32, tm_i = tmem + 128 + lane_addr + e0, tm_o = tmem + 256 + lane_addr + e0,
                 tm_s = tmem + 384 + lane_addr + e0;
  const float qscale = rsqrtf((float)D);
  const int chunks = live ? (rows + ML_CHUNK - 1) / ML_CHUNK : 0;
  bool ok = true;

  // ---- log gates of a chunk: the threads of the last column group request one token each ...
  float gi = 0.f, gf = 0.f;
  auto request_gates = [&](int t0) {
    const int t = t0 + tid - 384;
    gi = gf = 0.f;
    if (tid >= 384 && t < rows) {
      gi = gates[(long long)t * p.ld_gates];
      gf = gates[(long long)t * p.ld_gates + p.heads];
    }
  };
  const float bi = p.gate_bias[h], bf = p.gate_bias[p.heads + h];
  auto log_gates = [&](int t0, int b) {               // ... leave their logarithms where a and M will be
    if (tid < 384) return;
    const bool there = t0 + tid - 384 < rows;
    sa[b * 128 + tid - 384] = there ? log_input_gate(gi + bi, p.cap) : ML_NEVER;
    sM[b * 128 + tid - 384] = there ? log_forget_gate(gf + bf, p.cap) : 0.f;
  };
  // ... and one warp turns them into a, M and m
  auto scan_gates = [&](int b, float m_prev) {
    const float4 li = *reinterpret_cast<const float4*>(sa + b * 128 + lane * 4), lf = *reinterpret_cast<const float4*>(sM + b * 128 + lane * 4);
    float a[4] = {li.x, li.y, li.z, li.w}, F[4] = {lf.x, lf.x + lf.y, lf.x + lf.y + lf.z, lf.x + lf.y + lf.z + lf.w};
    float run = F[3];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += x;
    }
    run -= F[3];                                      // forget gates of the lanes before
    float top = ML_NEVER;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      F[j] += run;
      a[j] = a[j] == ML_NEVER ? ML_NEVER : a[j] - F[j];
      top = fmaxf(top, a[j]);
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, top, o);
      if (lane >= o) top = fmaxf(top, x);
    }
    top = __shfl_up_sync(0xffffffffu, top, 1);
    float M = lane == 0 ? m_prev : fmaxf(m_prev, top);
    float4 am, Mm, mm;
    M = fmaxf(M, a[0]); am.x = a[0] * LOG2E; Mm.x = M * LOG2E; mm.x = F[0] + M;
    M = fmaxf(M, a[1]); am.y = a[1] * LOG2E; Mm.y = M * LOG2E; mm.y = F[1] + M;
    M = fmaxf(M, a[2]); am.z = a[2] * LOG2E; Mm.z = M * LOG2E; mm.z = F[2] + M;
    M = fmaxf(M, a[3]); am.w = a[3] * LOG2E; Mm.w = M * LOG2E; mm.w = F[3] + M;
    *reinterpret_cast<float4*>(sa + b * 128 + lane * 4) = am;
    *reinterpret_cast<float4*>(sM + b * 128 + lane * 4) = Mm;
    *reinterpret_cast<float4*>(sm + b * 128 + lane * 4) = mm;
    if (lane == 0) sprev[b] = m_prev * LOG2E;
  };
  // S: columns [e0, e0 + HE) of row r; split into shared memory, times g in tensor memory
  auto publish_state = [&](const float (&s)[HE], float g) __attribute__((always_inline)) {
    uint32_t raw[HE];
#pragma unroll
    for (int i = 0; i < HE; ++i) raw[i] = __float_as_uint(s[i] * g);
    ml_tmem_st<HE>(tm_s, raw);
#pragma unroll
    for (int q = 0; q < HE / 8; ++q) {
      float f[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = r < D ? s[q * 8 + i] : 0.f;
      uint4 hi, lo;
      ml_split8(f, hi, lo);
      const uint32_t at = ml_swz(r, e0 / 8 + q);
      *reinterpret_cast<uint4*>(smem + L::OFF_SH + at) = hi;
      *reinterpret_cast<uint4*>(smem + L::OFF_SL + at) = lo;
    }
  };
  // q, k, v of the chunk at row t: 64-column panels, swizzled like the operands
  auto load_chunk = [&](int t) {
    const int pd = (D + 63) / 64, pe = (E + 63) / 64;
    mbar_expect_tx(bar_l, (uint32_t)(2 * pd + pe) * 16384u);
    for (int i = 0; i < pd; ++i) {
      tma_load_2d(smem + L::OFF_Q + i * 16384, &tm_proj, bar_l, h * D + i * 64, row0 + t);
      tma_load_2d(smem + L::OFF_K + i * 16384, &tm_proj, bar_l, p.heads * D + h * D + i * 64, row0 + t);
    }
    for (int i = 0; i < pe; ++i)
      tma_load_2d(smem + L::OFF_V + i * 16384, &tm_proj, bar_l, 2 * p.heads * D + h * E + i * 64, row0 + t);
  };
  if (issuer && chunks > 0 && elect_one()) load_chunk(0);
  __syncwarp();
  if (chunks > 0) {
    request_gates(0);
    log_gates(0, 0);
    request_gates(ML_CHUNK);
  }
  __syncthreads();
  if (issuer && chunks > 0) scan_gates(0, pos0 > 0 ? state_n[D] : 0.f);
  __syncthreads();
  if (chunks > 0) {
    if (tid < 128) sn[tid] = pos0 > 0 && tid < D ? state_n[tid] : 0.f;
    float s[HE];
#pragma unroll
    for (int i = 0; i < HE; ++i) s[i] = (pos0 > 0 && r < D && e0 + i < E) ? state[(long long)r * E + e0 + i] : 0.f;
    publish_state(s, ml_exp2(sprev[0] - sM[127]));
    tmem_st_wait();
  }
  const int kp = D / 8, k_step = ML_THREADS / kp, k_t = tid / kp, k_c8 = tid - k_t * kp;     // a thread's pieces of K
  const int ksteps = (D + 15) / 16;

  for (int ch = 0; ch < chunks; ++ch) {
    const int t0 = ch * ML_CHUNK, n = min(ML_CHUNK, rows - t0), b = ch & 1;
    const uint32_t ph = ch & 1;
    const bool last = ch + 1 == chunks;
    const float *a_b = sa + b * 128, *M_b = sM + b * 128;
    if (!mbar_wait(bar_l, ph, abort_word)) { ok = false; *abort_word = ERR_WAIT_FULL; }
    if ((D & 15) && cg == 0)                          // columns past dim that the last step of the products touches
      *reinterpret_cast<uint4*>(smem + L::OFF_Q + ml_swz(r, D / 8)) = make_uint4(0, 0, 0, 0);
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();

    if (issuer) {
      if (elect_one()) {
        tc_fence_after();
        constexpr uint32_t id_qk = make_idesc_bf16(128, 128, false, false);
        constexpr uint32_t id_xv = make_idesc_bf16(128, EP, false, true);
        auto kstep = [](int k) { return (uint32_t)(((k / 4) * 16384 + (k % 4) * 32) >> 4); };
        const uint64_t q = make_smem_desc(smem_u32(smem + L::OFF_Q), 16, 1024), k = make_smem_desc(smem_u32(smem + L::OFF_K), 16, 1024);
        const uint64_t sh = make_smem_desc(smem_u32(smem + L::OFF_SH), 16384, 1024);
        const uint64_t sl = make_smem_desc(smem_u32(smem + L::OFF_SL), 16384, 1024);
        for (int i = 0; i < ksteps; ++i) umma_f16_ss(tmem, q + kstep(i), k + kstep(i), id_qk, i ? 1u : 0u);
        umma_commit(bar_a);
        mbar_expect_tx(bar_g, (uint32_t)((E + 63) / 64) * 16384u);
        for (int i = 0; i < (E + 63) / 64; ++i)
          tma_load_2d(smem + L::OFF_KL + i * 16384, &tm_proj, bar_g, 2 * p.heads * D + p.heads * E + h * E + i * 64, row0 + t0);
        for (int i = 0; i < ksteps; ++i) umma_f16_ss(tmem + 128, q + kstep(i), sh + (uint32_t)(i * 128), id_xv, i ? 1u : 0u);
        for (int i = 0; i < ksteps; ++i) umma_f16_ss(tmem + 128, q + kstep(i), sl + (uint32_t)(i * 128), id_xv, 1u);
      }
      __syncwarp();
    }
    if (!last) {                                      // the gates of the next chunk
      log_gates(t0 + ML_CHUNK, b ^ 1);
      request_gates(t0 + 2 * ML_CHUNK);
    }
    const float M_end = M_b[127], M_r = M_b[r];
    const float c_r = ml_exp2(sprev[b] - M_r);        // how much of the earlier state row r still sees
    // ---- q_t . n_prev, a quarter of the dims per thread
    float den = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c8 = cg * 4 + i;
      if (c8 * 8 >= D) break;
      float f[8];
      ml_unpack8(*reinterpret_cast<const uint4*>(smem + L::OFF_Q + ml_swz(r, c8)), f);
      const float4 n0 = *reinterpret_cast<const float4*>(sn + c8 * 8), n1 = *reinterpret_cast<const float4*>(sn + c8 * 8 + 4);
      den += (f[0] * n0.x + f[1] * n0.y) + (f[2] * n0.z + f[3] * n0.w) + (f[4] * n1.x + f[5] * n1.y) + (f[6] * n1.z + f[7] * n1.w);
    }
    den *= c_r;
    // ---- scores -> weighted, causal, split; back to tensor memory as the A operand of P V, each group over its own columns
    if (!mbar_wait(bar_a, ph, abort_word)) { ok = false; *abort_word = ERR_WAIT_MISC; }
    tc_fence_after();
    {
      uint32_t hi[16], lo[16];
      if (cg > quarter) {                             // every key lies behind every row
#pragma unroll
        for (int i = 0; i < 16; ++i) hi[i] = lo[i] = 0u;
      } else {
        uint32_t s[32];
        tmem_ld_32x32(tm_a, s);
        tmem_ld_wait();
        const bool edge = cg == quarter;
        float den1 = 0.f;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float2 av = *reinterpret_cast<const float2*>(a_b + cg * 32 + 2 * i);
          float x = __uint_as_float(s[2 * i]) * ml_exp2(av.x - M_r), y = __uint_as_float(s[2 * i + 1]) * ml_exp2(av.y - M_r);
          if (edge) {
            x = 2 * i <= lane ? x : 0.f;
            y = 2 * i + 1 <= lane ? y : 0.f;
          }
          den += x;
          den1 += y;
          ml_split2(x, y, hi[i], lo[i]);
        }
        den += den1;
      }
      tmem_st_32x16(tm_a, hi);
      tmem_st_32x16(tm_a + 16, lo);
    }
    sden[cg * 128 + r] = den;
    if (!mbar_wait(bar_g, ph, abort_word)) { ok = false; *abort_word = ERR_WAIT_MISC; }
    uint4 gate[HE / 8];
#pragma unroll
    for (int q = 0; q < HE / 8; ++q) gate[q] = *reinterpret_cast<const uint4*>(smem + L::OFF_KL + ml_swz(r, e0 / 8 + q));
    tmem_st_wait();
    tc_fence_before();
    __syncthreads();
    if (issuer) {
      if (elect_one()) {
        tc_fence_after();
        constexpr uint32_t id_xv = make_idesc_bf16(128, EP, false, true);
        const uint64_t v = make_smem_desc(smem_u32(smem + L::OFF_V), 16384, 1024);
#pragma unroll
        for (int part = 0; part < 2; ++part)             // O_intra = P V
#pragma unroll
          for (int k = 0; k < 8; ++k)
            umma_f16_ts(tmem + 256, tmem + (k / 2) * 32 + part * 16 + (k % 2) * 8, v + (uint32_t)(k * 128), id_xv, (part | k) ? 1u : 0u);
        umma_commit(bar_o);
      }
      __syncwarp();
    }
    // ---- K~: weighted rows, split in place (hi) and beside (lo); their column sums for n
    if (k_t < k_step) {
      float col[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
      for (int t = k_t; t < ML_CHUNK; t += k_step) {
        const float w = ml_exp2(a_b[t] - M_end);
        const uint32_t at = ml_swz(t, k_c8);
        float f[8];
        ml_unpack8(*reinterpret_cast<const uint4*>(smem + L::OFF_K + at), f);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          f[i] = t < n ? f[i] * w : 0.f;
          col[i] += f[i];
        }
        uint4 hi, lo;
        ml_split8(f, hi, lo);
        *reinterpret_cast<uint4*>(smem + L::OFF_K + at) = hi;
        *reinterpret_cast<uint4*>(smem + L::OFF_KL + at) = lo;
      }
      *reinterpret_cast<float4*>(scol + k_t * D + k_c8 * 8) = make_float4(col[0], col[1], col[2], col[3]);
      *reinterpret_cast<float4*>(scol + k_t * D + k_c8 * 8 + 4) = make_float4(col[4], col[5], col[6], col[7]);
    }
    fence_proxy_async_smem();
    __syncthreads();
    if (issuer) {
      if (elect_one()) {
        tc_fence_after();
        constexpr uint32_t id_kv = make_idesc_bf16(128, EP, true, true);
        const uint64_t v = make_smem_desc(smem_u32(smem + L::OFF_V), 16384, 1024);
        const uint64_t kh = make_smem_desc(smem_u32(smem + L::OFF_K), 16384, 1024), kl = make_smem_desc(smem_u32(smem + L::OFF_KL), 16384, 1024);
#pragma unroll
        for (int part = 0; part < 2; ++part)             // S = g S_prev + K~^T V
#pragma unroll
          for (int k = 0; k < 8; ++k)
            umma_f16_ss(tmem + 384, (part ? kl : kh) + (uint32_t)(k * 128), v + (uint32_t)(k * 128), id_kv, 1u);
        umma_commit(bar_s);
      }
      __syncwarp();
      if (!last) scan_gates(b ^ 1, sm[b * 128 + 127]);
    }
    // ---- n
    if (tid < D) {
      float s = ml_exp2(sprev[b] - M_end) * sn[tid], s1 = 0.f;
      int i = 0;
      for (; i + 1 < k_step; i += 2) {
        s += scol[i * D + tid];
        s1 += scol[(i + 1) * D + tid];
      }
      if (i < k_step) s += scol[i * D + tid];
      s += s1;
      sn[tid] = s;
      if (last && ok) state_n[tid] = s;
    }
    if (last && tid == 0 && ok) state_n[D] = sm[b * 128 + 127];
    // ---- outputs of this thread's row and columns: both parts, the normaliser, the sum of squares
    if (!mbar_wait(bar_o, ph, abort_word)) { ok = false; *abort_word = ERR_WAIT_MISC; }
    tc_fence_after();
    float o[HE];
    {
      const float d4 = fabsf(((sden[r] + sden[128 + r]) + (sden[256 + r] + sden[384 + r])) * qscale);
      const float low = qscale / (fmaxf(d4, expf(-sm[b * 128 + r])) + 1e-6f), ci = c_r * low;
      uint32_t x[HE], y[HE];
      ml_tmem_ld<HE>(tm_i, x);
      ml_tmem_ld<HE>(tm_o, y);
      tmem_ld_wait();
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < HE; ++i) {
        o[i] = fmaf(__uint_as_float(x[i]), ci, __uint_as_float(y[i]) * low);
        if (e0 + i < E) ss = fmaf(o[i], o[i], ss);
      }
      srms[cg * 128 + r] = ss;
    }
    tc_fence_before();
    __syncthreads();
    // ---- state and outputs once the last product is done
    if (!mbar_wait(bar_s, ph, abort_word)) { ok = false; *abort_word = ERR_WAIT_MISC; }
    tc_fence_after();
    if (issuer && !last) {                              // every MMA of this chunk is done: its operands can be replaced
      if (elect_one()) load_chunk(t0 + ML_CHUNK);
      __syncwarp();
    }
    {
      const float inv = rsqrtf(((srms[r] + srms[128 + r]) + (srms[256 + r] + srms[384 + r])) / (float)E + p.eps);
#pragma unroll
      for (int q = 0; q < HE / 8; ++q) {
        float g[8];
        ml_unpack8(gate[q], g);
        const float4 w0 = *reinterpret_cast<const float4*>(sw + e0 + q * 8), w1 = *reinterpret_cast<const float4*>(sw + e0 + q * 8 + 4);
        const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
        for (int i = 0; i < 8; ++i) g[i] = o[q * 8 + i] * (inv * w[i]) * ml_sigmoid(g[i]);
        *reinterpret_cast<uint4*>(smem + L::OFF_KL + ml_swz(r, e0 / 8 + q)) =
            make_uint4(pack_bf16x2(g[0], g[1]), pack_bf16x2(g[2], g[3]), pack_bf16x2(g[4], g[5]), pack_bf16x2(g[6], g[7]));
      }
    }
    // ---- state: keep it for the next chunk, or leave it in the slot after the last one
    uint32_t raw[HE];
    ml_tmem_ld<HE>(tm_s, raw);
    tmem_ld_wait();
    if (last) {
      if (r < D && ok) {
#pragma unroll
        for (int q = 0; q < HE / 4; ++q)
          if (e0 + q * 4 < E)                            // vdim is a multiple of 8
            *reinterpret_cast<float4*>(state + (long long)r * E + e0 + q * 4) =
                make_float4(__uint_as_float(raw[q * 4]), __uint_as_float(raw[q * 4 + 1]), __uint_as_float(raw[q * 4 + 2]),
                            __uint_as_float(raw[q * 4 + 3]));
      }
    } else {
      float s[HE];
#pragma unroll
      for (int i = 0; i < HE; ++i) s[i] = __uint_as_float(raw[i]);
      publish_state(s, ml_exp2(sprev[b ^ 1] - sM[(b ^ 1) * 128 + 127]));
      tmem_st_wait();
    }
    __syncthreads();
    for (int i = tid; i < n * (EP / 8); i += ML_THREADS) {
      const int t = i / (EP / 8), c8 = i % (EP / 8);
      if (c8 * 8 < E)
        *reinterpret_cast<uint4*>(gy + (long long)(t0 + t) * p.ld_y + c8 * 8) = *reinterpret_cast<const uint4*>(smem + L::OFF_KL + ml_swz(t, c8));
    }
  }
  if (!live) {
    for (int t = warp; t < rows; t += ML_THREADS / 32)
      for (int c = lane * 8; c < E; c += 256) *reinterpret_cast<uint4*>(gy + (long long)t * p.ld_y + c) = make_uint4(0, 0, 0, 0);
  }
  tc_fence_before();
  __syncthreads();
  if (*abort_word != 0) {
    if (tid == 0 && p.status != nullptr) atomicCAS(p.status, 0u, (*abort_word) | (blockIdx.x << 8));
    const uint64_t w0 = globaltimer_ns();
    while (globaltimer_ns() - w0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

template <int EP>
static int launch_mlstm_chunk(const CUtensorMap& tm, const MlstmParams& p, cudaStream_t st) {
  auto kern = mlstm_chunk_kernel<EP>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, MlstmSmem<EP>::TOTAL) != cudaSuccess) return -3;
    configured = true;
  }
  launch_dep(kern, p.seqs * p.heads, ML_THREADS, MlstmSmem<EP>::TOTAL, st, tm, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace b200

using namespace b200;

// See MlstmParams.  f32 != 0: activations are fp32, else bf16.  chunked != 0: the tensor-core kernel (bf16, cu given, dim and vdim
// multiples of 8 up to 128).
extern "C" int b200_mlstm(const void* proj, long long ld_proj, const float* gates, long long ld_gates, const void* h, long long ld_h,
                          const void* w_gates, long long ld_wg, int width, const float* gate_bias, const void* weight, void* y, long long ld_y, float* state, const int* state_slots, const int* cu,
                          const int* positions, int seqs, int rows, int heads, int dim, int vdim, int stride, int num_slots,
                          float cap, float eps, int f32, int chunked, uint32_t* status, cudaStream_t st) {
  if (seqs <= 0 || rows <= 0) return 0;
  if (heads <= 0 || dim <= 0 || vdim <= 0 || heads > 65535 || stride < dim * vdim + dim + 1 || stride % 4 || !(cap > 0.f)) return -10;
  MlstmParams p;
  p.proj = proj; p.ld_proj = ld_proj; p.gates = gates; p.ld_gates = ld_gates; p.h = h; p.ld_h = ld_h; p.w_gates = w_gates;
  p.ld_wg = ld_wg; p.width = width; p.gate_bias = gate_bias; p.weight = weight;
  p.y = y; p.ld_y = ld_y; p.state = state; p.state_slots = state_slots; p.cu = cu; p.positions = positions; p.seqs = seqs;
  p.rows = rows; p.heads = heads; p.dim = dim; p.vdim = vdim; p.stride = stride; p.num_slots = num_slots; p.cap = cap;
  p.eps = eps; p.status = status;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(state);
  if (chunked) {
    if (f32 || cu == nullptr || gates == nullptr || dim > 128 || vdim > 128 || dim % 8 || vdim % 8) return -11;
    if (ld_proj % 8 || ld_y % 8 || (ptrs | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(weight)) & 15) return -11;
    CUtensorMap tm;
    if (make_tmap_bf16_2d(&tm, proj, (uint64_t)rows, (uint64_t)2 * heads * (dim + vdim), (uint64_t)ld_proj, 64, ML_CHUNK)) return -20;
    return vdim <= 64 ? launch_mlstm_chunk<64>(tm, p, st) : launch_mlstm_chunk<128>(tm, p, st);
  }
  const bool vec = vdim % 4 == 0 && ld_proj % 4 == 0 && (2 * heads * dim) % 4 == 0 && (ptrs & 15) == 0;
  const int groups = vec ? vdim / 4 : vdim;
  const int rg = groups < 256 ? 256 / groups : 1;
  const size_t smem = (2ull * dim + (size_t)rg * vdim) * sizeof(float);
  if (smem > 48 * 1024) return -12;
  const bool step = vec && cu == nullptr && groups <= 256 && (dim + rg - 1) / rg <= 16 && (dim & 1) == 0;
  if (gates == nullptr && (!step || h == nullptr || w_gates == nullptr || width <= 0 || ld_h % 4 || ld_wg % 4 ||
                           (reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(w_gates)) & 15))
    return -13;
  if (step) {
    const unsigned blocks = (unsigned)((long long)seqs * heads);
    const bool small = (dim + rg - 1) / rg <= 4;
    if (f32) {
      if (small) launch_dep(mlstm_step_kernel<float, 4>, blocks, 256, smem, st, p);
      else launch_dep(mlstm_step_kernel<float, 16>, blocks, 256, smem, st, p);
    } else {
      if (small) launch_dep(mlstm_step_kernel<__nv_bfloat16, 4>, blocks, 256, smem, st, p);
      else launch_dep(mlstm_step_kernel<__nv_bfloat16, 16>, blocks, 256, smem, st, p);
    }
    return cudaGetLastError() == cudaSuccess ? 0 : -4;
  }
  const dim3 grid(seqs, heads);
  if (f32) {
    if (vec) launch_dep(mlstm_recurrent_kernel<float, 4>, grid, 256, smem, st, p);
    else launch_dep(mlstm_recurrent_kernel<float, 1>, grid, 256, smem, st, p);
  } else {
    if (vec) launch_dep(mlstm_recurrent_kernel<__nv_bfloat16, 4>, grid, 256, smem, st, p);
    else launch_dep(mlstm_recurrent_kernel<__nv_bfloat16, 1>, grid, 256, smem, st, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
