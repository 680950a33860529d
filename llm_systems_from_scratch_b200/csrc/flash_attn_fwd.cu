// Causal FlashAttention forward for sm_100a, reading Q, K and V directly out of the packed
// (batch*seq, 3*H*dh) QKV activation (no head transposes) and writing O as (batch*seq, H*dh).
// Replaces the library SDPA call of the reference (llm-core/llm_core/model.py:381-382) and its
// naive masked-softmax path (model.py:308-325).
//
// One CTA owns TWO 128-query tiles (A, B) of one (batch, head) and walks the key/value tiles up to the
// diagonal.  The two tiles take turns on the tensor pipe, so the softmax of one overlaps the MMAs of the other:
//   warp 0      TMA producer: Q_A, Q_B once, then K_j / V_j into two-stage rings (128B swizzle)
//   warp 1      MMA issuer:   S_X = Q_X K_j^T (TMEM, 128 fp32 columns per tile)  and  O_X += P_X V_j
//   warps 2-5   softmax of tile A, warps 6-9 softmax of tile B: one thread per query row, no exchange between
//               threads.  Two passes over the row in tensor memory (row max, then exp2 / sum / bf16 pack); P is
//               written back over the S columns it came from (tcgen05.st) and is the A operand of the P V MMA
//               straight from tensor memory.  O is rescaled in TMEM only when the running max moved by more
//               than 2^8 (vote per warp).
// Tensor-pipe order per key tile j: P_A V_j, S_A(j+1), P_B V_j, S_B(j+1).
//
// WINDOW instances (b200_flash_window_fwd) serve portions of prompts under a sliding window: queries and keys come from
// separate matrices, a sequence has more keys than queries (the earlier tokens its first queries can still see), tile X
// walks only the key tiles its window touches, and the epilogue can multiply with sigmoid(gate), element by element or per head.
// ROPE instances have one more 64-column panel of queries and keys: rotated parts, whose keys are shared by all heads and come from a
// matrix of their own.  With heads of 128 the second stage of values makes room for them.
#include "ptx.cuh"

namespace b200 {

int make_tmap_bf16_2d(CUtensorMap* tm, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_cols,
                      uint32_t box_rows);

__device__ __forceinline__ float fa_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ float fa_sigmoid(float g) {     // (1 + tanh(g / 2)) / 2, one special-function instruction
  float t;
  asm("tanh.approx.f32 %0, %1;" : "=f"(t) : "f"(0.5f * g));
  return fmaf(0.5f, t, 0.5f);
}

__device__ __forceinline__ float fmax3(float a, float b, float c) {
  float r;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c));
  return r;
}

// 2^x on the FMA and integer pipes (no special-function unit): round x to the nearest integer n with the
// 1.5 * 2^23 trick, evaluate a cubic on the remainder in [-0.5, 0.5] (relative error 8e-5, far below bf16
// rounding of the result) and add n to the exponent field.  x must be <= 127; x below -126 gives 2^-126.
__device__ __forceinline__ float fa_exp2_poly(float x) {
  x = fmaxf(x, -126.f);
  const float t = x + 12582912.f;
  const float f = x - (t - 12582912.f);
  float pl = fmaf(f, 0.05508868f, 0.24260405f);
  pl = fmaf(pl, f, 0.69327624f);
  pl = fmaf(pl, f, 0.99992894f);
  return __int_as_float(__float_as_int(pl) + (__float_as_int(t) << 23));
}

// Packed fp32 pairs: one FMA-pipe instruction for two elements.
__device__ __forceinline__ void fma2(float& d0, float& d1, float a0, float a1, float b, float c) {
  asm("{\n\t"
      ".reg .b64 ra, rb, rc, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\t"
      "mov.b64 rb, {%4, %4};\n\t"
      "mov.b64 rc, {%5, %5};\n\t"
      "fma.rn.f32x2 rd, ra, rb, rc;\n\t"
      "mov.b64 {%0, %1}, rd;\n\t"
      "}"
      : "=f"(d0), "=f"(d1)
      : "f"(a0), "f"(a1), "f"(b), "f"(c));
}
__device__ __forceinline__ void add2(float& d0, float& d1, float a0, float a1) {   // (d0, d1) += (a0, a1)
  asm("{\n\t"
      ".reg .b64 ra, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\t"
      "mov.b64 rd, {%0, %1};\n\t"
      "add.rn.f32x2 rd, rd, ra;\n\t"
      "mov.b64 {%0, %1}, rd;\n\t"
      "}"
      : "+f"(d0), "+f"(d1)
      : "f"(a0), "f"(a1));
}

constexpr int FA_POLY_PER_8 = 0;   // of every 8 exponentials, this many are evaluated by fa_exp2_poly

constexpr int FA_BQ = 128;   // queries per tile (two tiles per CTA)
constexpr int FA_BK = 128;   // keys per step
constexpr int FA_THREADS = 64 + 256;   // TMA warp, MMA warp, 4 + 4 softmax warps

struct FlashFwdParams {
  __nv_bfloat16* o;      // (rows, d)
  float* lse;            // (batch, heads, seq)
  const int* cu_seqlens; // optional (batch+1) row offsets for packed variable-length sequences
  int batch, seq, heads, d;  // d = heads * dh; seq = max sequence length when cu_seqlens is given
  int n_qblk;            // 128-query tiles per sequence; a CTA takes two of them
  float scale_log2;      // softmax scale * log2(e)
  uint32_t* status;
  // WINDOW instances only
  const int* cu_k;       // (batch+1) row offsets of the keys; queries are the last positions of their sequence's keys
  int window;            // a query sees the `window` keys up to and including its own position
  int dim, vdim;         // columns of a head's queries and keys; columns that are written (<= DH)
  int q_step, k_step, v_step, v_off;    // columns from head to head of queries, keys, values; first column of the values
  int head_gate;         // gate has one column per head
  int rot, qr_col, qr_step, kr_col;     // ROPE: columns of the rotated part, where they are in the queries and in tm_kr
  long long ld_o;
  const __nv_bfloat16* gate;   // optional (rows, heads * vdim), row pitch ld_gate
  long long ld_gate;
  int out_vec, gate_vec; // 16-byte stores / loads are possible
  long long* trace;      // optional timeline of CTA `trace_cta` (tuning aid); null = off
  int trace_cta;
};

// stamp[(role * 64 + step) * 8 + slot] = SM clock, written by one lane of the traced CTA
#define FWD_TRACE(role, step, slot)                                                          \
  do {                                                                                       \
    if (p.trace != nullptr && (int)blockIdx.x == p.trace_cta && lane == 0 && (step) < 64)    \
      p.trace[((role) * 64 + (step)) * 8 + (slot)] = clock64();                              \
  } while (0)

template <int DH, bool ROPE>
struct FlashFwdSmem {
  static constexpr int PANELS = DH / 64;              // 64-column (128-byte) panels per tile
  static constexpr int TILE_BYTES = 128 * DH * 2;     // V tile
  static constexpr int QK_BYTES = TILE_BYTES + (ROPE ? 16384 : 0);      // Q or K tile
  static constexpr int V_STAGES = ROPE && DH == 128 ? 1 : 2;
  static constexpr int OFF_Q = 0;                     // Q_A, Q_B
  static constexpr int OFF_K = OFF_Q + 2 * QK_BYTES;
  static constexpr int OFF_V = OFF_K + 2 * QK_BYTES;
  static constexpr int OFF_BAR = OFF_V + V_STAGES * TILE_BYTES;
  static constexpr int NUM_BARS = 1 + 4 + 4 + 2 + 4 + 2;  // q, k full/empty, v full/empty, s_full[2], p_full[2][2], o_full[2]
  static constexpr int TOTAL = OFF_BAR + NUM_BARS * 8 + 16 + 1024;
};

template <int DH, bool WINDOW, bool ROPE>
__global__ void __launch_bounds__(FA_THREADS, 1)
flash_fwd_kernel(const __grid_constant__ CUtensorMap tm_qkv, const __grid_constant__ CUtensorMap tm_kv,
                 const __grid_constant__ CUtensorMap tm_kr, const FlashFwdParams p) {
  static_assert(WINDOW || !ROPE, "");
  using L = FlashFwdSmem<DH, ROPE>;
  constexpr int VS = L::V_STAGES;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;    // [2]
  uint64_t* k_empty = bars + 3;   // [2]  both tiles' S MMAs on this K stage have been issued and completed
  uint64_t* v_full = bars + 5;    // [2]
  uint64_t* v_empty = bars + 7;   // [2]  both tiles' P V MMAs on this V stage have completed
  uint64_t* s_full = bars + 9;    // [2]  per tile: S_X(j) is in tensor memory (and P_X V_{j-1} has completed)
  uint64_t* p_full = bars + 11;   // [2][2]  per tile and half of the key tile: P_X(j) is in tensor memory (128 arrivals)
  uint64_t* o_full = bars + 15;   // [2]  per tile: the last P V MMA has completed
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + L::NUM_BARS);
  volatile uint32_t* abort_word = tmem_holder + 1;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  // Work assignment: longest-first over the whole grid (latest query tiles = most key steps), so the tail of the
  // launch is made of short CTAs; the (b, h) index varies fastest.
  const int n_pair = (p.n_qblk + 1) >> 1;
  const int bh = blockIdx.x % (p.batch * p.heads);
  const int pair = n_pair - 1 - blockIdx.x / (p.batch * p.heads);
  const int b = bh / p.heads, h = bh % p.heads;
  int row_base, seq_len;
  if (p.cu_seqlens != nullptr) {
    row_base = p.cu_seqlens[b];
    seq_len = p.cu_seqlens[b + 1] - row_base;
  } else {
    row_base = b * p.seq;
    seq_len = p.seq;
  }
  int key_base = row_base, shift = 0;      // first key row; position of query 0 among the keys
  if (WINDOW) {
    key_base = p.cu_k[b];
    shift = p.cu_k[b + 1] - key_base - seq_len;
  }
  // CTA-uniform tile geometry: tile X covers queries [q0[X], q0[X] + 128) and key tiles lo_t[X] .. n_kv_t[X] - 1.  Tile A's
  // range starts and ends no later than tile B's and the two ranges leave no gap, so the CTA walks lo_t[0] .. n_kv - 1.
  const int q0_t[2] = {pair * 2 * FA_BQ, pair * 2 * FA_BQ + FA_BQ};
  int n_kv_t[2], lo_t[2];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    n_kv_t[x] = q0_t[x] < seq_len ? (min(q0_t[x] + FA_BQ, seq_len) + shift + FA_BK - 1) / FA_BK : 0;
    lo_t[x] = (WINDOW && n_kv_t[x] > 0) ? max(0, q0_t[x] + shift - p.window + 1) / FA_BK : 0;
  }
  const int n_kv = max(n_kv_t[0], n_kv_t[1]);
  const int j0 = lo_t[0];
  const bool active = n_kv > 0;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[2 * i], 128);
      mbar_init(&p_full[2 * i + 1], 128);
      mbar_init(&o_full[i], 1);
    }
    *abort_word = 0;
    fence_barrier_init();
    prefetch_tensormap(&tm_qkv);
    if (WINDOW) prefetch_tensormap(&tm_kv);
    if (ROPE) prefetch_tensormap(&tm_kr);
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;
  // columns: S_A [0,128)  S_B [128,256)  O_A [256,256+DH)  O_B [384,384+DH); P_X overlays the first 64 columns of S_X

  const int col_q = h * (WINDOW ? p.q_step : DH), col_k = WINDOW ? h * p.k_step : p.d + h * DH,
            col_v = WINDOW ? p.v_off + h * p.v_step : 2 * p.d + h * DH;
  const int pd = WINDOW ? (p.dim + 63) / 64 : L::PANELS;                // panels of queries and keys that are loaded
  const int ksteps = WINDOW ? (p.dim + 15) / 16 : DH / 16;
  const CUtensorMap* const map_kv = WINDOW ? &tm_kv : &tm_qkv;

  if (warp == 0) {
    if (active && elect_one()) {   // elect.sync keeps the issuing code warp-uniform (descriptors in uniform registers)
      // rows past the end of the tensor are zero-filled by TMA; rows of a following packed sequence are masked or unused
      const uint32_t qk_bytes = (uint32_t)(pd + (ROPE ? 1 : 0)) * 16384u;
      mbar_expect_tx(q_full, 2 * qk_bytes);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
#pragma unroll
        for (int pn = 0; pn < L::PANELS; ++pn)
          if (pn < pd)
            tma_load_2d(smem + L::OFF_Q + x * L::QK_BYTES + pn * 16384, &tm_qkv, q_full, col_q + pn * 64, row_base + q0_t[x]);
        if (ROPE)
          tma_load_2d(smem + L::OFF_Q + x * L::QK_BYTES + L::TILE_BYTES, &tm_qkv, q_full, p.qr_col + h * p.qr_step, row_base + q0_t[x]);
      }
      for (int j = j0; j < n_kv; ++j) {
        const int st = (j - j0) & 1;
        const uint32_t ph = ((j - j0) >> 1) & 1;
        const int krow = key_base + j * FA_BK;
        if (!mbar_wait(&k_empty[st], ph ^ 1, abort_word)) { *abort_word = ERR_WAIT_EMPTY; break; }
        mbar_expect_tx(&k_full[st], qk_bytes);
#pragma unroll
        for (int pn = 0; pn < L::PANELS; ++pn)
          if (pn < pd)
            tma_load_2d(smem + L::OFF_K + st * L::QK_BYTES + pn * 16384, map_kv, &k_full[st], col_k + pn * 64, krow);
        if (ROPE) tma_load_2d(smem + L::OFF_K + st * L::QK_BYTES + L::TILE_BYTES, &tm_kr, &k_full[st], p.kr_col, krow);
        const int sv = (j - j0) % VS;
        if (!mbar_wait(&v_empty[sv], (((j - j0) / VS) & 1) ^ 1, abort_word)) { *abort_word = ERR_WAIT_EMPTY; break; }
        mbar_expect_tx(&v_full[sv], L::TILE_BYTES);
#pragma unroll
        for (int pn = 0; pn < L::PANELS; ++pn)
          tma_load_2d(smem + L::OFF_V + sv * L::TILE_BYTES + pn * 16384, map_kv, &v_full[sv], col_v + pn * 64, krow);
      }
    }
  } else if (warp == 1) {
    if (active && elect_one()) {
      const int lane = 0;   // the tracing macro stamps from the issuing thread
      (void)lane;
      constexpr uint32_t idesc_qk = make_idesc_bf16(128, FA_BK, false, false);
      constexpr uint32_t idesc_pv = make_idesc_bf16(128, DH, false, true);
      auto issue_s = [&](int x, int j) {   // S_X(j) = Q_X K_j^T
        const uint64_t q_desc = make_smem_desc(smem_u32(smem + L::OFF_Q + x * L::QK_BYTES), 16, 1024);
        const uint64_t k_desc = make_smem_desc(smem_u32(smem + L::OFF_K + ((j - j0) & 1) * L::QK_BYTES), 16, 1024);
        if (ROPE) {
          const int rsteps = (p.rot + 15) / 16;
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            if (k >= rsteps) break;
            const uint32_t off = (L::TILE_BYTES + k * 32) >> 4;
            umma_f16_ss(tmem_base + x * 128, q_desc + off, k_desc + off, idesc_qk, k > 0 ? 1u : 0u);
          }
        }
#pragma unroll
        for (int k = 0; k < DH / 16; ++k) {
          if (WINDOW && k >= ksteps) break;
          const uint32_t off = ((k / 4) * 16384 + (k % 4) * 32) >> 4;
          umma_f16_ss(tmem_base + x * 128, q_desc + off, k_desc + off, idesc_qk, (ROPE || k > 0) ? 1u : 0u);
        }
        umma_commit(&s_full[x]);
      };
      // O_X += P_X(j) V_j, one half of the key tile at a time (the softmax warps publish P in two halves):
      // A = P from tensor memory (16 keys = 8 packed columns), B = V MN-major (dh contiguous, keys are rows of
      // 128 B): 16 keys = 2048 B; dh panels 16384 B apart.
      auto issue_pv = [&](int x, int j, int half) {
        const uint64_t v_desc = make_smem_desc(smem_u32(smem + L::OFF_V + ((j - j0) % VS) * L::TILE_BYTES), 16384, 1024);
#pragma unroll
        for (int kk = 0; kk < FA_BK / 32; ++kk) {
          const int k = half * (FA_BK / 32) + kk;
          umma_f16_ts(tmem_base + 256 + x * 128, tmem_base + x * 128 + k * 8, v_desc + ((k * 2048) >> 4), idesc_pv,
                      (j > lo_t[x] || k > 0) ? 1u : 0u);
        }
        if (half == 1 && j == n_kv_t[x] - 1) umma_commit(&o_full[x]);
      };
      bool ok = mbar_wait(q_full, 0, abort_word) && mbar_wait(&k_full[0], 0, abort_word);
      if (ok) {
        tc_fence_after();
        if (n_kv_t[0] > 0) issue_s(0, j0);
        if (n_kv_t[1] > 0 && lo_t[1] == j0) issue_s(1, j0);
        umma_commit(&k_empty[0]);
      }
      for (int j = j0; j < n_kv && ok; ++j) {
        const int st = (j - j0) & 1, sv = (j - j0) % VS;
        const uint32_t pv = ((j - j0) / VS) & 1;
        bool v_ready = false, k_ready = false;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          if (j >= lo_t[x] && j < n_kv_t[x]) {
            ok = mbar_wait(&p_full[2 * x], (j - lo_t[x]) & 1, abort_word) && (v_ready || mbar_wait(&v_full[sv], pv, abort_word));
            if (!ok) break;
            v_ready = true;
            tc_fence_after();
            FWD_TRACE(1, j, x * 4 + 0);
            issue_pv(x, j, 0);
            ok = mbar_wait(&p_full[2 * x + 1], (j - lo_t[x]) & 1, abort_word);
            if (!ok) break;
            tc_fence_after();
            issue_pv(x, j, 1);
            FWD_TRACE(1, j, x * 4 + 1);
          }
          if (x == 1) umma_commit(&v_empty[sv]);   // both tiles are done with V_j
          if (j + 1 >= lo_t[x] && j + 1 < n_kv_t[x]) {
            ok = k_ready || mbar_wait(&k_full[st ^ 1], ((j + 1 - j0) >> 1) & 1, abort_word);
            if (!ok) break;
            k_ready = true;
            tc_fence_after();
            issue_s(x, j + 1);
            FWD_TRACE(1, j, x * 4 + 2);
          }
        }
        if (ok && j + 1 < n_kv) umma_commit(&k_empty[st ^ 1]);   // both tiles are done with K_{j+1}
      }
      if (!ok) *abort_word = ERR_WAIT_FULL;
    }
  } else if (active) {
    // ----------------------------------------------------------------- softmax warps: one thread per query row
    const int x = (warp - 2) >> 2;              // tile A (warps 2-5) or B (warps 6-9)
    const int quarter = warp & 3;               // TMEM lanes [32*quarter, 32*quarter+32) are visible to this warp
    const int r = quarter * 32 + lane;          // row inside the query tile
    const int q0 = (pair * 2 + x) * FA_BQ;
    const int n_kv_x = x == 0 ? n_kv_t[0] : n_kv_t[1];
    const int lo_x = x == 0 ? lo_t[0] : lo_t[1];
    const int q_idx = q0 + r;                   // query of this thread
    const int q_key = q_idx + shift;            // its position among the keys
    const int q_low = WINDOW ? q_key - p.window : -1;   // the last key it no longer sees
    const uint32_t lane_addr = uint32_t(quarter * 32) << 16;
    const uint32_t tm_s = tmem_base + x * 128 + lane_addr;
    const uint32_t tm_o = tmem_base + 256 + x * 128 + lane_addr;
    float m_run = -INFINITY;                    // running reference max in scaled log2 units
    float l_run = 0.f;                          // running row sum relative to m_run
    bool ok = true;
    if (WINDOW && p.gate != nullptr && !p.head_gate && q_idx < seq_len) {      // the epilogue's gate row into L2
      const __nv_bfloat16* grow = p.gate + (long long)(row_base + q_idx) * p.ld_gate + h * p.vdim;
      for (int i = 0; i < p.vdim; i += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(grow + i));
    }
    for (int j = lo_x; j < n_kv_x; ++j) {
      const int trole = warp;
      FWD_TRACE(trole, j, 0);
      if (!mbar_wait(&s_full[x], (j - lo_x) & 1, abort_word)) { ok = false; break; }
      tc_fence_after();
      FWD_TRACE(trole, j, 1);
      const int k0 = j * FA_BK;
      // tile touches the diagonal or the lower edge of the window (warp-uniform)
      const bool diag = (k0 + FA_BK - 1 > q0 + shift) || (WINDOW && k0 <= q0 + FA_BQ - 1 + shift - p.window);
      // pass 1: row maximum over the raw scores (the softmax scale is positive, so it is applied afterwards).
      // The load of chunk c+1 is in flight while chunk c is reduced.
      float mx = -INFINITY;
      // Key k0 + e is visible iff e - first <= span as unsigned numbers (one comparison for both edges of the window).
      const int first = q_low + 1 - k0;
      const uint32_t span = WINDOW ? (uint32_t)(p.window - 1) : 0u;
      auto hidden = [&](int e) { return WINDOW ? (uint32_t)(e - first) > span : k0 + e > q_key; };
      auto row_max = [&](const bool masked) __attribute__((always_inline)) {
        uint32_t sa[32], sb[32];
        tmem_ld_32x32(tm_s, sa);
        tmem_ld_wait();
#pragma unroll
        for (int c = 0; c < FA_BK / 32; ++c) {
          uint32_t (&cur)[32] = (c & 1) ? sb : sa;
          uint32_t (&nxt)[32] = (c & 1) ? sa : sb;
          if (c + 1 < FA_BK / 32) tmem_ld_32x32(tm_s + (c + 1) * 32, nxt);
          if (masked) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (hidden(c * 32 + i)) cur[i] = 0xff800000u;   // -inf
          }
#pragma unroll
          for (int i = 0; i < 32; i += 2) mx = fmax3(mx, __uint_as_float(cur[i]), __uint_as_float(cur[i + 1]));
          if (c + 1 < FA_BK / 32) tmem_ld_wait();
        }
      };
      if (WINDOW) {                    // two copies: tiles inside the window pay nothing for its edges
        if (diag) row_max(true);
        else row_max(false);
      } else {
        row_max(diag);
      }
      mx *= p.scale_log2;
      FWD_TRACE(trole, j, 2);
      // Lazy rescale: keep the old reference max unless it moved by more than 8 (a factor 256).
      float m_new = m_run;
      if (mx > m_run + 8.f) m_new = mx;
      const bool need = m_new != m_run;
      const float alpha = (m_run == -INFINITY) ? 0.f : fa_exp2(m_run - m_new);
      // S_X(j) was issued after P_X V_{j-1}, so that MMA has completed and O_X may be rescaled here.
      if (j > lo_x && __any_sync(0xffffffffu, need)) {
        const float f = need ? alpha : 1.f;
#pragma unroll 1
        for (int c = 0; c < DH / 32; ++c) {
          uint32_t o[32];
          tmem_ld_32x32(tm_o + c * 32, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
          tmem_st_32x32(tm_o + c * 32, o);
        }
      }
      FWD_TRACE(trole, j, 3);
      // pass 2: P = exp2(S * scale - m), row sum, bf16 pack; P chunk c (16 packed columns) lands on S columns
      // [16c, 16c+16), all of which this thread has already read.
      // (a row whose window starts in a later tile has seen no key yet: every P is masked to zero below)
      const float m_ref = (WINDOW && m_new == -INFINITY) ? 0.f : m_new;
      float sum = 0.f, sum1 = 0.f;
      auto weights = [&](const bool masked) __attribute__((always_inline)) {
        uint32_t sa[32], sb[32];
        tmem_ld_32x32(tm_s, sa);
        tmem_ld_wait();
#pragma unroll
        for (int c = 0; c < FA_BK / 32; ++c) {
          uint32_t (&s)[32] = (c & 1) ? sb : sa;
          uint32_t (&nxt)[32] = (c & 1) ? sa : sb;
          uint32_t pk[16];
          if (c + 1 < FA_BK / 32) tmem_ld_32x32(tm_s + (c + 1) * 32, nxt);   // in flight while this chunk is processed
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            float x0, x1;
            fma2(x0, x1, __uint_as_float(s[i]), __uint_as_float(s[i + 1]), p.scale_log2, -m_ref);
            float e0 = ((i & 7) < FA_POLY_PER_8) ? fa_exp2_poly(x0) : fa_exp2(x0);
            float e1 = (((i + 1) & 7) < FA_POLY_PER_8) ? fa_exp2_poly(x1) : fa_exp2(x1);
            if (masked) {
              e0 = hidden(c * 32 + i) ? 0.f : e0;
              e1 = hidden(c * 32 + i + 1) ? 0.f : e1;
            }
            add2(sum, sum1, e0, e1);
            pk[i / 2] = pack_bf16x2(e0, e1);
          }
          if (c + 1 < FA_BK / 32) tmem_ld_wait();   // before the store below: wait::ld covers the prefetched chunk
          tmem_st_32x16(tm_s + c * 16, pk);
          if (c == 1 || c == 3) {   // publish this half of P
            tmem_st_wait();
            tc_fence_before();
            mbar_arrive(&p_full[2 * x + (c >> 1)]);
          }
        }
      };
      if (WINDOW) {
        if (diag) weights(true);
        else weights(false);
      } else {
        weights(diag);
      }
      l_run = l_run * (need ? alpha : 1.f) + (sum + sum1);
      m_run = m_new;
      FWD_TRACE(trole, j, 4);
    }
    // ------------------------------------------------------------------- epilogue
    if (ok && n_kv_x > 0) ok = mbar_wait(&o_full[x], 0, abort_word);
    if (ok && n_kv_x > 0) {
      tc_fence_after();
      float inv_l = 1.f / l_run;
      const bool valid = q_idx < seq_len;
      if (WINDOW && p.head_gate && valid) inv_l *= fa_sigmoid(__bfloat162float(p.gate[(long long)(row_base + q_idx) * p.ld_gate + h]));
      __nv_bfloat16* orow = WINDOW ? p.o + (long long)(row_base + q_idx) * p.ld_o + h * p.vdim
                                   : p.o + (size_t)(row_base + q_idx) * p.d + h * DH;
#pragma unroll 1
      for (int c = 0; c < DH / 32; ++c) {
        uint32_t o[32];
        tmem_ld_32x32(tm_o + c * 32, o);
        tmem_ld_wait();
        if (WINDOW) {
          if (valid && c * 32 < p.vdim) {      // no early continue: the next tensor-memory load needs the whole warp
            const __nv_bfloat16* grow =
                p.gate != nullptr && !p.head_gate ? p.gate + (long long)(row_base + q_idx) * p.ld_gate + h * p.vdim + c * 32 : nullptr;
            const int n = min(32, p.vdim - c * 32);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
              if (q * 8 >= n) break;
              float f[8];
#pragma unroll
              for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(o[q * 8 + i]) * inv_l;
              if (grow != nullptr && p.gate_vec && q * 8 + 8 <= n) {
                const uint4 gv = *reinterpret_cast<const uint4*>(grow + q * 8);
                const uint32_t gg[4] = {gv.x, gv.y, gv.z, gv.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                  const float2 g2 = unpack_bf16x2(gg[i]);
                  f[2 * i] *= fa_sigmoid(g2.x);
                  f[2 * i + 1] *= fa_sigmoid(g2.y);
                }
              } else if (grow != nullptr) {
#pragma unroll
                for (int i = 0; i < 8; ++i)
                  if (q * 8 + i < n) f[i] *= fa_sigmoid(__bfloat162float(grow[q * 8 + i]));
              }
              if (p.out_vec && q * 8 + 8 <= n) {
                *reinterpret_cast<uint4*>(orow + c * 32 + q * 8) =
                    make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
              } else {
#pragma unroll
                for (int i = 0; i < 8; ++i)
                  if (q * 8 + i < n) orow[c * 32 + q * 8 + i] = __float2bfloat16(f[i]);
              }
            }
          }
        } else if (valid) {
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            uint4 v = make_uint4(pack_bf16x2(__uint_as_float(o[q * 8 + 0]) * inv_l, __uint_as_float(o[q * 8 + 1]) * inv_l),
                                 pack_bf16x2(__uint_as_float(o[q * 8 + 2]) * inv_l, __uint_as_float(o[q * 8 + 3]) * inv_l),
                                 pack_bf16x2(__uint_as_float(o[q * 8 + 4]) * inv_l, __uint_as_float(o[q * 8 + 5]) * inv_l),
                                 pack_bf16x2(__uint_as_float(o[q * 8 + 6]) * inv_l, __uint_as_float(o[q * 8 + 7]) * inv_l));
            *reinterpret_cast<uint4*>(orow + c * 32 + q * 8) = v;
          }
        }
      }
      if (valid && p.lse != nullptr)
        p.lse[((size_t)b * p.heads + h) * p.seq + q_idx] = (m_run + log2f(l_run)) * 0.6931471805599453f;
    } else if (!ok && lane == 0) {
      *abort_word = ERR_WAIT_TMEM_FULL;
    }
  }

  __syncwarp();
  tc_fence_before();
  __syncthreads();
  if (*abort_word != 0) {
    if (threadIdx.x == 0 && p.status != nullptr) atomicCAS(p.status, 0u, (*abort_word) | (blockIdx.x << 8));
    const uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

template <int DH, bool WINDOW, bool ROPE = false>
static int launch_flash_fwd(const CUtensorMap& tm, const CUtensorMap& tm_kv, const FlashFwdParams& p, cudaStream_t stream,
                            const CUtensorMap* tm_kr = nullptr) {
  using L = FlashFwdSmem<DH, ROPE>;
  auto kern = flash_fwd_kernel<DH, WINDOW, ROPE>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL) != cudaSuccess) return -3;
    configured = true;
  }
  const int grid = p.batch * p.heads * ((p.n_qblk + 1) / 2);   // one CTA per pair of query tiles
  kern<<<grid, FA_THREADS, L::TOTAL, stream>>>(tm, tm_kv, tm_kr != nullptr ? *tm_kr : tm_kv, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace b200

using namespace b200;

static long long* g_fwd_trace = nullptr;
static int g_fwd_trace_cta = 0;

// Tuning aid: record the timeline of CTA `cta` of the next forward launches into `buf`
// (device memory, 10 roles x 64 steps x 8 stamps of 8 bytes); null switches it off.
extern "C" void b200_flash_fwd_set_trace(long long* buf, int cta) {
  g_fwd_trace = buf;
  g_fwd_trace_cta = cta;
}

// qkv: (rows, 3*heads*dh) bf16 row-major, rows = batch*seq (or cu_seqlens[batch] when packed).
// o: (rows, heads*dh) bf16.  lse: (batch, heads, seq) fp32 or null.  dh must be 64 or 128.
extern "C" int b200_flash_fwd(const void* qkv, void* o, float* lse, int batch, int seq, int heads, int dh,
                              float scale, uint32_t* status, cudaStream_t stream) {
  if (dh != 64 && dh != 128) return -10;
  if (reinterpret_cast<uintptr_t>(qkv) & 15 || reinterpret_cast<uintptr_t>(o) & 15) return -10;
  if (batch <= 0 || seq <= 0) return 0;
  const int d = heads * dh;
  CUtensorMap tm;
  if (make_tmap_bf16_2d(&tm, qkv, (uint64_t)batch * seq, (uint64_t)3 * d, (uint64_t)3 * d, 64, 128)) return -20;
  FlashFwdParams p = {};
  p.o = (__nv_bfloat16*)o; p.lse = lse; p.cu_seqlens = nullptr;
  p.batch = batch; p.seq = seq; p.heads = heads; p.d = d;
  p.n_qblk = (seq + FA_BQ - 1) / FA_BQ;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.status = status;
  p.trace = g_fwd_trace; p.trace_cta = g_fwd_trace_cta;
  return dh == 64 ? launch_flash_fwd<64, false>(tm, tm, p, stream) : launch_flash_fwd<128, false>(tm, tm, p, stream);
}

// Packed variable-length sequences (serving prefill): cu_seqlens (batch+1) int32 on the device,
// total_rows = cu_seqlens[batch], max_seq = longest sequence.
extern "C" int b200_flash_varlen_fwd(const void* qkv, void* o, const int* cu_seqlens, int batch, int max_seq,
                                     int total_rows, int heads, int dh, float scale, uint32_t* status,
                                     cudaStream_t stream) {
  if (dh != 64 && dh != 128) return -10;
  if (reinterpret_cast<uintptr_t>(qkv) & 15 || reinterpret_cast<uintptr_t>(o) & 15) return -10;
  if (batch <= 0 || total_rows <= 0) return 0;
  const int d = heads * dh;
  CUtensorMap tm;
  if (make_tmap_bf16_2d(&tm, qkv, (uint64_t)total_rows, (uint64_t)3 * d, (uint64_t)3 * d, 64, 128)) return -20;
  FlashFwdParams p = {};
  p.o = (__nv_bfloat16*)o; p.lse = nullptr; p.cu_seqlens = cu_seqlens;
  p.batch = batch; p.seq = max_seq; p.heads = heads; p.d = d;
  p.n_qblk = (max_seq + FA_BQ - 1) / FA_BQ;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.status = status;
  p.trace = g_fwd_trace; p.trace_cta = g_fwd_trace_cta;
  return dh == 64 ? launch_flash_fwd<64, false>(tm, tm, p, stream) : launch_flash_fwd<128, false>(tm, tm, p, stream);
}

// Portions of prompts under a sliding window.  q: (total_q, q_cols), kv: (total_k, kv_cols); a head's queries, keys and values are dim,
// dim and vdim columns (at most 128; more than 64 take the instance for 128) at h * q_step, h * k_step and v_off + h * v_step (steps and
// offsets multiples of 8).  Columns are loaded in boxes of 64 and multiplied 16 at a time: up to the next multiple of 16 they must be
// finite, and zero in q or k.  cu_q / cu_k: (batch + 1) row offsets on the device; query i of a sequence with Lq queries and Lk keys
// sits at key position i + Lk - Lq and sees the `window` keys up to it (window <= 0: all of them).
// rot > 0 (at most 64): the score gains rotated parts, rot columns of q at qr_col + h * qr_step and of kr (total_k, kr_cols) at kr_col,
// the latter for all heads; the same rules.
// o: (total_q, heads * vdim), row pitch ld_o, multiplied by sigmoid(gate) when gate is given: (total_q, heads * vdim), or
// (total_q, heads) with head_gate.  scale must be positive.
struct FlashWindowShape {        // passed by pointer through the C interface: the field order is part of it
  long long ld_q, ld_kv, ld_kr, ld_o, ld_gate;
  int q_cols, kv_cols, kr_cols, heads, dim, vdim, q_step, k_step, v_step, v_off, rot, qr_col, qr_step, kr_col, window, head_gate;
  float scale;
};

extern "C" int b200_flash_window_fwd(const void* q, const void* kv, const void* kr, void* o, const void* gate, const int* cu_q,
                                     const int* cu_k, int batch, int max_q, int total_q, int total_k, const FlashWindowShape* s,
                                     uint32_t* status, cudaStream_t stream) {
  const int dh = s->dim > 64 || s->vdim > 64 ? 128 : 64;
  if (s->heads <= 0 || s->dim <= 0 || s->dim > 128 || s->vdim <= 0 || s->vdim > 128 || !(s->scale > 0.f)) return -10;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(kr)) & 15 || s->ld_q % 8 ||
      s->ld_kv % 8 || (s->q_step | s->k_step | s->v_step | s->v_off) % 8)
    return -10;
  if (s->rot < 0 || s->rot > 64 || (s->rot > 0 && (kr == nullptr || s->ld_kr % 8 || (s->qr_col | s->qr_step | s->kr_col) % 8))) return -10;
  if (batch <= 0 || total_q <= 0) return 0;
  CUtensorMap tm, tm_kv, tm_kr;
  if (make_tmap_bf16_2d(&tm, q, (uint64_t)total_q, (uint64_t)s->q_cols, (uint64_t)s->ld_q, 64, 128)) return -20;
  if (make_tmap_bf16_2d(&tm_kv, kv, (uint64_t)total_k, (uint64_t)s->kv_cols, (uint64_t)s->ld_kv, 64, 128)) return -21;
  if (s->rot > 0 && make_tmap_bf16_2d(&tm_kr, kr, (uint64_t)total_k, (uint64_t)s->kr_cols, (uint64_t)s->ld_kr, 64, 128)) return -22;
  FlashFwdParams p = {};
  p.o = (__nv_bfloat16*)o; p.cu_seqlens = cu_q; p.cu_k = cu_k;
  p.batch = batch; p.seq = max_q; p.heads = s->heads; p.d = s->heads * dh;
  p.n_qblk = (max_q + FA_BQ - 1) / FA_BQ;
  p.scale_log2 = s->scale * 1.4426950408889634f;
  p.window = s->window > 0 ? s->window : (1 << 30);
  p.dim = s->dim; p.vdim = s->vdim; p.q_step = s->q_step; p.k_step = s->k_step; p.v_step = s->v_step; p.v_off = s->v_off;
  p.rot = s->rot; p.qr_col = s->qr_col; p.qr_step = s->qr_step; p.kr_col = s->kr_col;
  p.ld_o = s->ld_o; p.gate = (const __nv_bfloat16*)gate; p.ld_gate = s->ld_gate; p.head_gate = gate != nullptr && s->head_gate;
  p.out_vec = s->vdim % 8 == 0 && s->ld_o % 8 == 0 && (reinterpret_cast<uintptr_t>(o) & 15) == 0;
  p.gate_vec = s->vdim % 8 == 0 && s->ld_gate % 8 == 0 && (reinterpret_cast<uintptr_t>(gate) & 15) == 0;
  p.status = status;
  if (s->rot > 0)
    return dh == 64 ? launch_flash_fwd<64, true, true>(tm, tm_kv, p, stream, &tm_kr) : launch_flash_fwd<128, true, true>(tm, tm_kv, p, stream, &tm_kr);
  return dh == 64 ? launch_flash_fwd<64, true>(tm, tm_kv, p, stream) : launch_flash_fwd<128, true>(tm, tm_kv, p, stream);
}
