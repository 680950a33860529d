// Retention: attention without softmax whose memory is a decaying matrix.  Per head S_t = decay S_(t-1) + k_t v_t^T and o_t = S_t^T q_t with
// rotated q, k (rotate-half pairs, 32-bit angles) and k scaled by dim^(-1/2); the output of a head is divided by its root
// mean square and multiplied by silu(gate).  The state (heads, dim, vdim) is fp32 and lives in a slot per request.
#include "typed.cuh"

namespace b200 {

int make_tmap_bf16_2d(CUtensorMap* tm, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_cols,
                      uint32_t box_rows);

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

// Decode step of a state that fits the block's registers (NR rows of four columns per thread): one block per (request,
// head), the whole state is requested before anything else, so the rotation, which needs little, runs under its latency.
template <typename T, int NR>
__global__ void __launch_bounds__(256, NR > 8 ? 2 : 3) retention_step_kernel(const RetentionParams p) {
  pdl_sync();
  extern __shared__ float rsm[];
  __shared__ float red[32];
  const int seq = blockIdx.x / p.heads, h = blockIdx.x - seq * p.heads;
  const int D = p.dim, E = p.vdim, groups = E / 4, rg = 256 / groups;
  float *qs = rsm, *ks = rsm + D, *part = rsm + 2 * D;         // [D], [D], [rg][E]
  const int ty = threadIdx.x / groups, tx = threadIdx.x - ty * groups;
  const int slot = p.state_slots[seq];
  const T* pr = reinterpret_cast<const T*>(p.proj) + (long long)seq * p.ld_proj;
  T* y = reinterpret_cast<T*>(p.y) + (long long)seq * p.ld_y + h * E;
  if (slot < 0 || slot >= p.num_slots) {
    if (slot >= p.num_slots && threadIdx.x == 0) report_bad_arg(p.status, 7);
    for (int c = threadIdx.x; c < E; c += 256) from_f(y[c], 0.f);
    return;
  }
  int pos = p.positions[seq];
  const bool on = ty < rg;
  float4* S = reinterpret_cast<float4*>(p.state + ((long long)slot * p.heads + h) * D * E) + tx;
  float4 s[NR];
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = ty + j * rg;
    s[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on && d < D && pos != 0) s[j] = __ldcs(S + (long long)d * groups);
  }
  const T* qr = pr + h * D;
  const T* kr = pr + p.heads * D + h * D;
  if (pos < 0 || (p.rot > 0 && pos >= p.ctx)) {
    if (threadIdx.x == 0) report_bad_arg(p.status, 8);
    pos = 0;
  }
  const int half = p.rot / 2;
  const float kscale = rsqrtf((float)D);
  for (int d = threadIdx.x; d < D; d += 256) {
    float qv = to_f(qr[d]), kv = to_f(kr[d]);
    if (d < p.rot) {
      const int i = d < half ? d : d - half, o = d < half ? d + half : d - half;
      const float c = p.cos_sin[(long long)pos * half + i];
      const float sn = d < half ? -p.cos_sin[((long long)p.ctx + pos) * half + i] : p.cos_sin[((long long)p.ctx + pos) * half + i];
      qv = qv * c + to_f(qr[o]) * sn;
      kv = kv * c + to_f(kr[o]) * sn;
    }
    qs[d] = qv;
    ks[d] = kv * kscale;
  }
  float v[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) load_vec<4>(pr + 2 * p.heads * D + h * E + tx * 4, v);
  const float decay = p.decay[h];
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = ty + j * rg;
    if (!on || d >= D) continue;
    const float kd = ks[d], qd = qs[d];
    s[j].x = fmaf(decay, s[j].x, kd * v[0]); s[j].y = fmaf(decay, s[j].y, kd * v[1]);
    s[j].z = fmaf(decay, s[j].z, kd * v[2]); s[j].w = fmaf(decay, s[j].w, kd * v[3]);
    o.x = fmaf(s[j].x, qd, o.x); o.y = fmaf(s[j].y, qd, o.y); o.z = fmaf(s[j].z, qd, o.z); o.w = fmaf(s[j].w, qd, o.w);
    __stcs(S + (long long)d * groups, s[j]);
  }
  if (on) *reinterpret_cast<float4*>(part + ty * E + tx * 4) = o;
  __syncthreads();
  float ss = 0.f, mine[4];
  int n = 0;
  for (int c = threadIdx.x; c < E && n < 4; c += 256, ++n) {           // E <= 1024
    float t = 0.f;
    for (int r = 0; r < rg; ++r) t += part[r * E + c];
    mine[n] = t;
    ss += t * t;
  }
  const float inv = rsqrtf(block_total(ss, red) / (float)E + p.eps);
  const T* gr = pr + 2 * p.heads * D + p.heads * E + h * E;
  n = 0;
  for (int c = threadIdx.x; c < E && n < 4; c += 256, ++n) {
    const float g = to_f(gr[c]);
    from_f(y[c], mine[n] * inv * (g / (1.f + __expf(-g))));
  }
}

// ------------------------------------------------------------------------------------ prompts, bf16, on the tensor cores
// One CTA = one (portion, head), chunks of n <= 128 tokens in order.  With r the last row of a chunk, scale the rotated
// rows in fp32:  q~_i = decay^(i-r) q_i,  k~_j = decay^(r-j) k_j  and let S' = decay^n S.  Then
//     O = causal(Q~ K~^T) V + Q~ S',        S <- S' + K~^T V,
// so the decays need no further work in the products.  What enters the recurrence keeps (close to) 32-bit precision:
// q~, k~, the scores and S' are each split into two bf16 parts (hi + lo, 16 significant bits) and the products of the
// parts are accumulated in fp32 (v is bf16 as projected); S itself stays fp32, in tensor memory between chunks.
//   tensor memory: scores [0, 128)  O [128, 128 + EP)  S [256, 256 + EP)  P hi [384, 448)  P lo [448, 512)
//   shared memory: Q~ hi, lo | K~ hi, lo | V | S' hi, lo, all 128-byte swizzled panels of 64 columns
// K~ and V serve two products each in the same storage (K-major and MN-major descriptors).
// Eight warps do the element-wise phases (two warps per 32 lanes of tensor memory, half of the columns each); a ninth
// issues TMA and MMAs, so that Q~ S' and the state's product run while the scores are masked and split.  TMA brings q, k
// and v of the next chunk while the outputs of this one are written: q and k land where their lo parts will be and are
// rotated, scaled and split in place (with shared memory full there is no L1 left that would hold loads in flight).
constexpr int RC_CHUNK = 128;
constexpr int RC_WORKERS = 256;
constexpr int RC_THREADS = RC_WORKERS + 32;

__device__ __forceinline__ void worker_barrier() { asm volatile("bar.sync 1, 256;" ::: "memory"); }   // RC_WORKERS threads

template <int EP>
struct RetChunkSmem {
  static constexpr int TILE = 32768;                 // 128 rows x 128 columns of bf16: two panels
  static constexpr int VT = EP / 64 * 16384;
  static constexpr int OFF_QH = 0, OFF_QL = TILE, OFF_KH = 2 * TILE, OFF_KL = 3 * TILE;
  static constexpr int OFF_V = 4 * TILE, OFF_SH = OFF_V + VT, OFF_SL = OFF_SH + VT;
  static constexpr int OFF_RMS = OFF_SL + VT;        // [2][128] floats
  static constexpr int OFF_POW = OFF_RMS + 1024;     // [129] floats
  static constexpr int OFF_BAR = OFF_POW + 520;
  static constexpr int TOTAL = OFF_BAR + 4 * 8 + 16 + 1024;
};

// 16-byte piece `c8` (8 columns) of row `r` in a tile of 64-column panels, 128-byte swizzle
__device__ __forceinline__ uint32_t swz(int r, int c8) {
  return (uint32_t)(c8 >> 3) * 16384u + (uint32_t)r * 128u + (uint32_t)(((c8 & 7) ^ (r & 7)) << 4);
}

__device__ __forceinline__ float silu_fast(float g) {      // g sigmoid(g) = g (1 + tanh(g / 2)) / 2
  float t;
  asm("tanh.approx.f32 %0, %1;" : "=f"(t) : "f"(0.5f * g));
  return 0.5f * g * (1.f + t);
}

// x = hi + lo with both parts bf16, eight values at a time
__device__ __forceinline__ void split8(const float (&x)[8], uint4& hi, uint4& lo) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    h[i] = pack_bf16x2(x[2 * i], x[2 * i + 1]);
    const float2 b = unpack_bf16x2(h[i]);
    l[i] = pack_bf16x2(x[2 * i] - b.x, x[2 * i + 1] - b.y);
  }
  hi = make_uint4(h[0], h[1], h[2], h[3]);
  lo = make_uint4(l[0], l[1], l[2], l[3]);
}
__device__ __forceinline__ void unpack8f(const uint4& v, float (&f)[8]) {
  const float2 a = unpack_bf16x2(v.x), b = unpack_bf16x2(v.y), c = unpack_bf16x2(v.z), d = unpack_bf16x2(v.w);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
}

template <int EP>
__global__ void __launch_bounds__(RC_THREADS, 1) retention_chunk_kernel(const __grid_constant__ CUtensorMap tm_proj, const RetentionParams p,
                                                                         const float* __restrict__ powers) {
  using L = RetChunkSmem<EP>;
  constexpr int HE = EP / 2;                          // columns of O and S that a thread handles
  extern __shared__ uint8_t rc_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(rc_raw) + 1023) & ~uintptr_t(1023));
  float* srms = reinterpret_cast<float*>(smem + L::OFF_RMS);
  float* spow = reinterpret_cast<float*>(smem + L::OFF_POW);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR);
  uint64_t *bar_a = bars, *bar_s = bars + 1, *bar_o = bars + 2, *bar_l = bars + 3;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + 4);
  volatile uint32_t* abort_word = tmem_holder + 1;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

  if (tid == 0) {
    for (int i = 0; i < 4; ++i) mbar_init(&bars[i], 1);
    *abort_word = 0;
    fence_barrier_init();
    prefetch_tensormap(&tm_proj);
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  for (int i = tid; i < (L::OFF_RMS >> 4); i += RC_THREADS) reinterpret_cast<uint4*>(smem)[i] = make_uint4(0, 0, 0, 0);
  pdl_sync();
  const int seq = blockIdx.x / p.heads, h = blockIdx.x - seq * p.heads;
  const int D = p.dim, E = p.vdim;
  for (int i = tid; i <= RC_CHUNK; i += RC_THREADS) spow[i] = powers[h * (RC_CHUNK + 1) + i];
  fence_proxy_async_smem();           // the zeros above come before what TMA writes
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;

  const int row0 = p.cu[seq], rows = p.cu[seq + 1] - row0;
  const int slot = p.state_slots[seq];
  const bool live = slot >= 0 && slot < p.num_slots;
  if (!live && slot >= p.num_slots && tid == 0) report_bad_arg(p.status, 10);
  const int pos0 = rows > 0 ? p.positions[row0] : 0;
  float* state = p.state + ((long long)(live ? slot : 0) * p.heads + h) * D * E;
  const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(p.proj) + (long long)row0 * p.ld_proj;
  const __nv_bfloat16* gg = proj + 2 * p.heads * D + p.heads * E + h * E;
  if (tid == 0 && live && p.rot > 0 && rows > 0 && pos0 + rows > p.ctx) report_bad_arg(p.status, 11);
  __nv_bfloat16* gy = reinterpret_cast<__nv_bfloat16*>(p.y) + (long long)row0 * p.ld_y + h * E;

  const int quarter = warp & 3, half = warp >> 2;
  const int r = quarter * 32 + lane;                  // this thread's row of tensor memory: a token, or a dim of S
  const uint32_t lane_addr = uint32_t(quarter * 32) << 16;
  const uint32_t tm_a = tmem + lane_addr, tm_o = tmem + 128 + lane_addr, tm_s = tmem + 256 + lane_addr,
                 tm_p = tmem + 384 + lane_addr;
  const int rot2 = p.rot / 2, n_rot = p.rot / 16, n_items = n_rot + (D - p.rot) / 8;
  const float kscale = rsqrtf((float)D);
  const int chunks = live ? (rows + RC_CHUNK - 1) / RC_CHUNK : 0;
  bool ok = true;

  // S' of the first chunk from the request's slot (the zero state at position 0)
  auto publish_state = [&](const float (&s)[32], int c) {       // columns [half * HE + 32 c, + 32) of row r
    uint32_t raw[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) raw[i] = __float_as_uint(s[i]);
    tmem_st_32x32(tm_s + half * HE + c * 32, raw);
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      float f[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = s[q * 8 + i];
      uint4 hi, lo;
      split8(f, hi, lo);
      const uint32_t at = swz(r, (half * HE + c * 32) / 8 + q);
      *reinterpret_cast<uint4*>(smem + L::OFF_SH + at) = hi;
      *reinterpret_cast<uint4*>(smem + L::OFF_SL + at) = lo;
    }
  };
  const bool worker = warp < RC_WORKERS / 32;
  // q, k, v of the chunk at row t: 64-column panels, swizzled like the operands; columns past the head are zeroed later
  auto load_chunk = [&](int t) {
    const int pd = (D + 63) / 64, pe = (E + 63) / 64;
    mbar_expect_tx(bar_l, (uint32_t)(2 * pd + pe) * 16384u);
    for (int i = 0; i < pd; ++i) {
      tma_load_2d(smem + L::OFF_QL + i * 16384, &tm_proj, bar_l, h * D + i * 64, row0 + t);
      tma_load_2d(smem + L::OFF_KL + i * 16384, &tm_proj, bar_l, p.heads * D + h * D + i * 64, row0 + t);
    }
    for (int i = 0; i < pe; ++i)
      tma_load_2d(smem + L::OFF_V + i * 16384, &tm_proj, bar_l, 2 * p.heads * D + h * E + i * 64, row0 + t);
  };
  if (!worker && chunks > 0 && elect_one()) load_chunk(0);
  __syncwarp();
  // Row-wise work: a thread owns one 16-byte piece (or one pair of rotated pieces) of rows t, t + step, ...
  const int vg = E / 8, v_step = RC_WORKERS / vg, v_t = tid / vg, v_c8 = tid - v_t * vg;
  const bool v_on = v_t < v_step;
  const int i_step = RC_WORKERS / n_items, i_t = tid / n_items, i_it = tid - i_t * n_items;
  const bool i_turn = i_it < n_rot;
  const int i_d0 = i_turn ? i_it * 8 : p.rot + (i_it - n_rot) * 8, i_d1 = i_turn ? i_d0 + rot2 : i_d0;
  if (worker && chunks > 0) {
    const float f = spow[min(rows, RC_CHUNK)];
#pragma unroll 1
    for (int c = 0; c < HE / 32; ++c) {
      float s[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        const int e = half * HE + c * 32 + i;
        s[i] = (pos0 > 0 && r < D && e < E) ? state[(long long)r * E + e] * f : 0.f;
      }
      publish_state(s, c);
    }
    tmem_st_wait();
  }

  for (int ch = 0; ch < chunks; ++ch) {
    const int t0 = ch * RC_CHUNK, n = min(RC_CHUNK, rows - t0);
    if (worker) {
      // ---- q~, k~: rotated, scaled, split; rows past the end become zero.  The angles of the first PRE rows are requested
      // before the wait: there is no L1 to speak of beside this much shared memory.
      constexpr int PRE = 4;
      float4 ang[PRE][4];                               // cos, cos, sin, sin
      auto load_angles = [&](int t, float4 (&a)[4]) {
        const float* cs = p.cos_sin + (long long)min(pos0 + t0 + min(t, n - 1), p.ctx - 1) * rot2 + i_d0;
        const float* sn = cs + (long long)p.ctx * rot2;
        a[0] = __ldg(reinterpret_cast<const float4*>(cs));
        a[1] = __ldg(reinterpret_cast<const float4*>(cs + 4));
        a[2] = __ldg(reinterpret_cast<const float4*>(sn));
        a[3] = __ldg(reinterpret_cast<const float4*>(sn + 4));
      };
#pragma unroll
      for (int j = 0; j < PRE; ++j) {
        ang[j][0] = ang[j][1] = make_float4(1.f, 1.f, 1.f, 1.f);
        ang[j][2] = ang[j][3] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i_turn && i_t < i_step && i_t + j * i_step < RC_CHUNK) load_angles(i_t + j * i_step, ang[j]);
      }
      if (!mbar_wait(bar_l, ch & 1, abort_word)) { ok = false; *abort_word = ERR_WAIT_FULL; }
      if (i_t < i_step) {
        auto item = [&](int t, const float4 (&an)[4]) __attribute__((always_inline)) {
          const float c[8] = {an[0].x, an[0].y, an[0].z, an[0].w, an[1].x, an[1].y, an[1].z, an[1].w};
          const float s[8] = {an[2].x, an[2].y, an[2].z, an[2].w, an[3].x, an[3].y, an[3].z, an[3].w};
          const float pw = t < n ? spow[n - 1 - t] : 1.f;
          const float fq = t < n ? __fdividef(1.f, pw) : 0.f, fk = t < n ? pw * kscale : 0.f;
          const uint32_t o0 = swz(t, i_d0 / 8), o1 = swz(t, i_d1 / 8);
          auto put = [&](float f, int off_hi, int off_lo) {
            float a[8], b2[8];
            unpack8f(*reinterpret_cast<const uint4*>(smem + off_lo + o0), a);
            unpack8f(*reinterpret_cast<const uint4*>(smem + off_lo + o1), b2);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              const float x = a[i], z = b2[i];
              a[i] = (x * c[i] - z * s[i]) * f;
              b2[i] = (z * c[i] + x * s[i]) * f;
            }
            uint4 hi, lo;
            split8(a, hi, lo);
            *reinterpret_cast<uint4*>(smem + off_hi + o0) = hi;
            *reinterpret_cast<uint4*>(smem + off_lo + o0) = lo;
            if (i_turn) {
              split8(b2, hi, lo);
              *reinterpret_cast<uint4*>(smem + off_hi + o1) = hi;
              *reinterpret_cast<uint4*>(smem + off_lo + o1) = lo;
            }
          };
          put(fq, L::OFF_QH, L::OFF_QL);
          put(fk, L::OFF_KH, L::OFF_KL);
        };
#pragma unroll
        for (int j = 0; j < PRE; ++j)
          if (i_t + j * i_step < RC_CHUNK) item(i_t + j * i_step, ang[j]);
#pragma unroll 1
        for (int t = i_t + PRE * i_step; t < RC_CHUNK; t += i_step) {
          float4 an[4];
          an[0] = an[1] = make_float4(1.f, 1.f, 1.f, 1.f);
          an[2] = an[3] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (i_turn) load_angles(t, an);
          item(t, an);
        }
      }
      for (int c8 = D / 8 + (tid >> 7); c8 < 16; c8 += 2) {          // columns past dim and vdim: neighbours' data
        const uint32_t at = swz(tid & 127, c8);
        *reinterpret_cast<uint4*>(smem + L::OFF_QH + at) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(smem + L::OFF_QL + at) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(smem + L::OFF_KH + at) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(smem + L::OFF_KL + at) = make_uint4(0, 0, 0, 0);
      }
      for (int c8 = E / 8 + (tid >> 7); c8 < EP / 8; c8 += 2)
        *reinterpret_cast<uint4*>(smem + L::OFF_V + swz(tid & 127, c8)) = make_uint4(0, 0, 0, 0);
    }
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();

    if (!worker && elect_one()) {
      tc_fence_after();
      constexpr uint32_t id_qk = make_idesc_bf16(128, 128, false, false);
      constexpr uint32_t id_xv = make_idesc_bf16(128, EP, false, true);
      constexpr uint32_t id_kv = make_idesc_bf16(128, EP, true, true);
      auto kmaj = [&](int off) { return make_smem_desc(smem_u32(smem + off), 16, 1024); };
      auto mnmaj = [&](int off) { return make_smem_desc(smem_u32(smem + off), 16384, 1024); };
      auto kstep = [](int k) { return (uint32_t)(((k / 4) * 16384 + (k % 4) * 32) >> 4); };
      const uint64_t qh = kmaj(L::OFF_QH), ql = kmaj(L::OFF_QL), kh = kmaj(L::OFF_KH), kl = kmaj(L::OFF_KL);
      const uint64_t v = mnmaj(L::OFF_V), sh = mnmaj(L::OFF_SH), sl = mnmaj(L::OFF_SL);
      const uint64_t kht = mnmaj(L::OFF_KH), klt = mnmaj(L::OFF_KL);
#pragma unroll
      for (int part = 0; part < 3; ++part)             // scores = Qh Kh^T + Qh Kl^T + Ql Kh^T
#pragma unroll
        for (int k = 0; k < 8; ++k)
          umma_f16_ss(tmem, (part == 2 ? ql : qh) + kstep(k), (part == 1 ? kl : kh) + kstep(k), id_qk, (part | k) ? 1u : 0u);
      umma_commit(bar_a);
#pragma unroll
      for (int part = 0; part < 3; ++part)             // O = Qh S'h + Qh S'l + Ql S'h
#pragma unroll
        for (int k = 0; k < 8; ++k)
          umma_f16_ss(tmem + 128, (part == 2 ? ql : qh) + kstep(k), (part == 1 ? sl : sh) + (uint32_t)(k * 128), id_xv,
                      (part | k) ? 1u : 0u);
#pragma unroll
      for (int part = 0; part < 2; ++part)             // S = S' + Kh^T V + Kl^T V
#pragma unroll
        for (int k = 0; k < 8; ++k)
          umma_f16_ss(tmem + 256, (part ? klt : kht) + (uint32_t)(k * 128), v + (uint32_t)(k * 128), id_kv, 1u);
      umma_commit(bar_s);
    }
    __syncwarp();
    const uint32_t ph = ch & 1;
    uint4 gate[EP / 16];
    if (worker) {
#pragma unroll
      for (int j = 0; j < EP / 16; ++j) {
        const int t = v_t + j * v_step;
        gate[j] = make_uint4(0, 0, 0, 0);
        if (v_on && t < n) gate[j] = *reinterpret_cast<const uint4*>(gg + (long long)(t0 + t) * p.ld_proj + v_c8 * 8);
      }
    // ---- scores -> causal, split, back to tensor memory as the A operand of P V
    if (!mbar_wait(bar_a, ph, abort_word)) { ok = false; *abort_word = ERR_WAIT_MISC; }
    tc_fence_after();
#pragma unroll 1
    for (int c = 0; c < 2; ++c) {
      uint32_t a[32];
      const int k0 = half * 64 + c * 32;
      tmem_ld_32x32(tm_a + k0, a);
      tmem_ld_wait();
      uint32_t hi[16], lo[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const float x = k0 + 2 * i <= r ? __uint_as_float(a[2 * i]) : 0.f;
        const float y = k0 + 2 * i + 1 <= r ? __uint_as_float(a[2 * i + 1]) : 0.f;
        hi[i] = pack_bf16x2(x, y);
        const float2 b = unpack_bf16x2(hi[i]);
        lo[i] = pack_bf16x2(x - b.x, y - b.y);
      }
      tmem_st_32x16(tm_p + half * 32 + c * 16, hi);
      tmem_st_32x16(tm_p + 64 + half * 32 + c * 16, lo);
    }
    tmem_st_wait();
    tc_fence_before();
    }
    __syncthreads();
    if (!worker && elect_one()) {
      tc_fence_after();
      constexpr uint32_t id_xv = make_idesc_bf16(128, EP, false, true);
      const uint64_t v = make_smem_desc(smem_u32(smem + L::OFF_V), 16384, 1024);
#pragma unroll
      for (int part = 0; part < 2; ++part)             // O += P V
#pragma unroll
        for (int k = 0; k < 8; ++k)
          umma_f16_ts(tmem + 128, tmem + 384 + part * 64 + k * 8, v + (uint32_t)(k * 128), id_xv, 1u);
      umma_commit(bar_o);
    }
    if (!worker) {
      if (ch + 1 < chunks) {                            // every MMA of this chunk is done: its operands can be replaced
        if (!mbar_wait(bar_o, ph, abort_word)) *abort_word = ERR_WAIT_MISC;
        if (elect_one()) load_chunk(t0 + RC_CHUNK);
      }
      __syncwarp();
      continue;
    }
    // ---- state: keep it for the next chunk, or leave it in the slot after the last one
    if (!mbar_wait(bar_s, ph, abort_word)) { ok = false; *abort_word = ERR_WAIT_MISC; }
    tc_fence_after();
    const bool last = ch + 1 == chunks;
    const float f = last ? 1.f : spow[min(RC_CHUNK, rows - t0 - RC_CHUNK)];
#pragma unroll 1
    for (int c = 0; c < HE / 32; ++c) {
      uint32_t raw[32];
      tmem_ld_32x32(tm_s + half * HE + c * 32, raw);
      tmem_ld_wait();
      if (last) {
        if (r < D && ok) {
#pragma unroll
          for (int q = 0; q < 8; ++q)
            if (half * HE + c * 32 + q * 4 < E)          // vdim is a multiple of 8
              *reinterpret_cast<float4*>(state + (long long)r * E + half * HE + c * 32 + q * 4) =
                  make_float4(__uint_as_float(raw[q * 4]), __uint_as_float(raw[q * 4 + 1]), __uint_as_float(raw[q * 4 + 2]),
                              __uint_as_float(raw[q * 4 + 3]));
        }
      } else {
        float s[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) s[i] = __uint_as_float(raw[i]) * f;
        publish_state(s, c);
      }
    }
    tmem_st_wait();
    // ---- output: root mean square of the head, gate, bf16
    if (!mbar_wait(bar_o, ph, abort_word)) { ok = false; *abort_word = ERR_WAIT_MISC; }
    tc_fence_after();
    uint32_t o[HE / 32][32];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < HE / 32; ++c) tmem_ld_32x32(tm_o + half * HE + c * 32, o[c]);
    tmem_ld_wait();
#pragma unroll
    for (int c = 0; c < HE / 32; ++c)
#pragma unroll
      for (int i = 0; i < 32; ++i) ss = fmaf(__uint_as_float(o[c][i]), __uint_as_float(o[c][i]), ss);
    srms[half * 128 + r] = ss;                          // columns beyond vdim are zero
    worker_barrier();
    const float inv = rsqrtf((srms[r] + srms[128 + r]) / (float)E + p.eps);
    // rows -> columns through shared memory (the tiles of the hi parts are free now, each half of the columns in one), so
    // that the gate and y move in whole rows
    constexpr int PIECES = EP / 8;                      // 16-byte pieces of half an fp32 row
    float4* stage = reinterpret_cast<float4*>(smem + (half ? L::OFF_KH : L::OFF_QH)) + r * PIECES;
#pragma unroll
    for (int c = 0; c < HE / 32; ++c)
#pragma unroll
      for (int q = 0; q < 8; ++q)
        stage[(c * 8 + q) ^ (r & (PIECES - 1))] =
            make_float4(__uint_as_float(o[c][q * 4]) * inv, __uint_as_float(o[c][q * 4 + 1]) * inv,
                        __uint_as_float(o[c][q * 4 + 2]) * inv, __uint_as_float(o[c][q * 4 + 3]) * inv);
    worker_barrier();
#pragma unroll
    for (int j = 0; j < EP / 16; ++j) {
      const int t = v_t + j * v_step;
      if (!v_on || t >= n) continue;
      const float4* from =
          reinterpret_cast<const float4*>(smem + (2 * v_c8 < PIECES ? L::OFF_QH : L::OFF_KH)) + t * PIECES;
      const int x = t & (PIECES - 1), pc = (2 * v_c8) & (PIECES - 1);
      const float4 y0 = from[pc ^ x], y1 = from[(pc + 1) ^ x];
      float g[8];
      unpack8f(gate[j], g);
#pragma unroll
      for (int i = 0; i < 8; ++i) g[i] = silu_fast(g[i]);
      *reinterpret_cast<uint4*>(gy + (long long)(t0 + t) * p.ld_y + v_c8 * 8) =
          make_uint4(pack_bf16x2(y0.x * g[0], y0.y * g[1]), pack_bf16x2(y0.z * g[2], y0.w * g[3]),
                     pack_bf16x2(y1.x * g[4], y1.y * g[5]), pack_bf16x2(y1.z * g[6], y1.w * g[7]));
    }
    worker_barrier();
    tc_fence_before();
  }
  if (!live) {
    for (int t = tid / 32; t < rows; t += RC_THREADS / 32)
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
static int launch_retention_chunk(const CUtensorMap& tm, const RetentionParams& p, const float* powers, cudaStream_t st) {
  auto kern = retention_chunk_kernel<EP>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, RetChunkSmem<EP>::TOTAL) != cudaSuccess) return -3;
    configured = true;
  }
  launch_dep(kern, p.seqs * p.heads, RC_THREADS, RetChunkSmem<EP>::TOTAL, st, tm, p, powers);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
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
  if (vec && cu == nullptr && groups <= 256 && (dim + rg - 1) / rg <= 16 && (dim & 3) == 0) {
    const long long blocks = (long long)seqs * heads;
    const bool small = (dim + rg - 1) / rg <= 4;
    if (f32) {
      if (small) launch_dep(retention_step_kernel<float, 4>, (unsigned)blocks, 256, smem, st, p);
      else launch_dep(retention_step_kernel<float, 16>, (unsigned)blocks, 256, smem, st, p);
    } else {
      if (small) launch_dep(retention_step_kernel<__nv_bfloat16, 4>, (unsigned)blocks, 256, smem, st, p);
      else launch_dep(retention_step_kernel<__nv_bfloat16, 16>, (unsigned)blocks, 256, smem, st, p);
    }
    return cudaGetLastError() == cudaSuccess ? 0 : -4;
  }
  if (f32) {
    if (vec) launch_dep(retention_recurrent_kernel<float, 4>, grid, 256, smem, st, p);
    else launch_dep(retention_recurrent_kernel<float, 1>, grid, 256, smem, st, p);
  } else {
    if (vec) launch_dep(retention_recurrent_kernel<__nv_bfloat16, 4>, grid, 256, smem, st, p);
    else launch_dep(retention_recurrent_kernel<__nv_bfloat16, 1>, grid, 256, smem, st, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// Prompts on the tensor cores (bf16): cu (seqs + 1) delimits the portions; `powers` (heads, 129) holds decay^m.  dim and vdim
// multiples of 8 up to 128, rot a multiple of 16, and decay^127 must stay well inside the range of bf16 exponents.
extern "C" int b200_retention_chunk(const void* proj, long long ld_proj, void* y, long long ld_y, float* state,
                                    const int* state_slots, const int* cu, const int* positions, const float* cos_sin,
                                    const float* powers, int seqs, int rows, int heads, int dim, int vdim, int rot, int ctx,
                                    int num_slots, float eps, uint32_t* status, cudaStream_t st) {
  if (seqs <= 0 || rows <= 0) return 0;
  if (heads <= 0 || dim <= 0 || vdim <= 0 || dim > 128 || vdim > 128 || dim % 8 || vdim % 8 || rot % 16 || rot < 0 ||
      rot > dim || cu == nullptr || powers == nullptr || (rot > 0 && cos_sin == nullptr))
    return -10;
  if (ld_proj % 8 || ld_y % 8 ||
      (reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(state) |
       reinterpret_cast<uintptr_t>(cos_sin)) & 15)
    return -11;
  RetentionParams p;
  p.proj = proj; p.ld_proj = ld_proj; p.y = y; p.ld_y = ld_y; p.state = state; p.state_slots = state_slots; p.cu = cu;
  p.positions = positions; p.cos_sin = cos_sin; p.decay = nullptr; p.seqs = seqs; p.rows = rows; p.heads = heads;
  p.dim = dim; p.vdim = vdim; p.rot = rot; p.ctx = ctx; p.num_slots = num_slots; p.eps = eps; p.status = status;
  CUtensorMap tm;
  if (make_tmap_bf16_2d(&tm, proj, (uint64_t)rows, (uint64_t)2 * heads * (dim + vdim), (uint64_t)ld_proj, 64, RC_CHUNK)) return -20;
  return vdim <= 64 ? launch_retention_chunk<64>(tm, p, powers, st) : launch_retention_chunk<128>(tm, p, powers, st);
}
