// Portions of prompts of grouped attention (see grouped_attention.cu) on tcgen05, keys and values straight from the paged cache.
//
// The pipeline is the FlashAttention kernel's (flash_attn_fwd.cu): one CTA owns two 128-query tiles A and B that take turns on the
// tensor pipe, scores and outputs in tensor memory, P over the scores, one thread per query row.
//   one map    A and B are consecutive query tiles of one head and share every key and value tile
//   two maps   A and B are the two maps of one query tile: each has its own keys, the values are shared, and the epilogue
//              takes the difference of both outputs, norms it per head and gates it
// Key tiles of 128 positions start at multiples of 128 and are copied as one TMA box per page and 64 columns (a box may bring
// columns of the next head: the query's pad is zero, and outputs past vdim are not stored).  Value rows past the request's
// last token are zeroed in shared memory before the product.
// A CTA walks the tiles of the kept first positions (both query tiles see them), then those of its window.
//   CAP   scores are capped softly in the second pass (the cap is monotone, so the row maximum is taken of the raw scores); a tile
//         whose scores stay below the cap evaluates tanh as a polynomial, others take capped_log2
//   SLOPE slope * distance comes off the scaled score in both passes (two fused multiply-adds per score, nothing is written back)
//   BIAS  a table per head and distance (shared memory) is added to the scaled scores, which go back to tensor memory for the
//         second pass; distances from the table's last entry on read that entry
#include "grouped_attention.cuh"

namespace b200 {

int make_tmap_bf16_2d(CUtensorMap* tm, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_cols,
                      uint32_t box_rows);

struct GroupedPrefillParams {
  __nv_bfloat16* o;
  const __nv_bfloat16* gate;    // optional
  long long ld_o, ld_gate;
  const float* bias;            // BIAS: (heads, bias_len)
  const int *cu, *positions, *tables;     // cu (portions + 1); positions per row; tables: line per portion
  int bias_len, portions, n_qblk, max_pages, page_size, num_pages;
  int out_vec, gate_vec;        // 16-byte stores / loads are possible
  float scale_log2;
  GroupedShape s;
  uint32_t* status;
};

constexpr int GP_THREADS = 64 + 256;      // TMA warp, MMA warp, 4 + 4 softmax warps
constexpr int GP_LUT_PAD = 254;           // table entries in front of distance 0 (keys of a tile that lie behind a query)

enum GroupedScores : int { SCORES_PLAIN = 0, SCORES_BIAS = 1, SCORES_CAP = 2, SCORES_SLOPE = 3 };

template <int P, bool BIAS>
struct GroupedPrefillSmem {
  static constexpr int TILE = 128 * 64 * P * 2;
  static constexpr int OFF_Q = 0, OFF_K = 2 * TILE, OFF_V = 4 * TILE;
  static constexpr int OFF_X = 6 * TILE;                   // exchange between the tiles: [2][2][128] floats
  static constexpr int OFF_BAR = OFF_X + 2048;
  static constexpr int NUM_BARS = 1 + 4 + 4 + 2 + 4 + 2;   // q, k full/empty, v full/empty, s_full[2], p_full[2][2], o_full[2]
  static constexpr int OFF_LUT = OFF_BAR + NUM_BARS * 8 + 16;
  static constexpr int total(int bias_len) { return OFF_LUT + (BIAS ? (bias_len + 2 * GP_LUT_PAD + 1) * 4 : 0) + 1024; }
};

__device__ __forceinline__ float gp_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gp_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gp_sigmoid(float g) {     // (1 + tanh(g / 2)) / 2, one special-function instruction
  float t;
  asm("tanh.approx.f32 %0, %1;" : "=f"(t) : "f"(0.5f * g));
  return fmaf(0.5f, t, 0.5f);
}
__device__ __forceinline__ float gp_max3(float a, float b, float c) {
  float r;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c));
  return r;
}
// packed fp32 pairs: (d0, d1) = (a0, a1) * b + c and (d0, d1) += (a0, a1)
__device__ __forceinline__ void gp_fma2(float& d0, float& d1, float a0, float a1, float b, float c) {
  asm("{\n\t.reg .b64 ra, rb, rc, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %4};\n\tmov.b64 rc, {%5, %5};\n\t"
      "fma.rn.f32x2 rd, ra, rb, rc;\n\tmov.b64 {%0, %1}, rd;\n\t}"
      : "=f"(d0), "=f"(d1)
      : "f"(a0), "f"(a1), "f"(b), "f"(c));
}
__device__ __forceinline__ void gp_add2(float& d0, float& d1, float a0, float a1) {
  asm("{\n\t.reg .b64 ra, rd;\n\tmov.b64 ra, {%2, %3};\n\tmov.b64 rd, {%0, %1};\n\t"
      "add.rn.f32x2 rd, rd, ra;\n\tmov.b64 {%0, %1}, rd;\n\t}"
      : "+f"(d0), "+f"(d1)
      : "f"(a0), "f"(a1));
}
// top tanh(z) - m for z = score * slope / (2 log2 e), |z| <= 1: tanh(z) = z Q(z^2), Q of degree 5 fitted by weighted least squares (error
// 3e-7).  k = z per score.
__device__ __forceinline__ void gp_tanh2(float& d0, float& d1, float s0, float s1, float k, float top, float m) {
  constexpr float c[6] = {0.99999684f, -0.33324003f, 0.13253525f, -0.050972860f, 0.016114177f, -0.0028394643f};
  const float2 z = __fmul2_rn(make_float2(s0, s1), make_float2(k, k));
  const float2 t = __fmul2_rn(z, z);
  float2 q = make_float2(c[5], c[5]);
#pragma unroll
  for (int i = 4; i >= 0; --i) q = __ffma2_rn(q, t, make_float2(c[i], c[i]));
  q = __fmul2_rn(q, z);
  q = __ffma2_rn(q, make_float2(top, top), make_float2(-m, -m));
  d0 = q.x;
  d1 = q.y;
}
__device__ __forceinline__ float gp_min3(float a, float b, float c) {
  float r;
  asm("min.f32 %0, %1, %2, %3;" : "=f"(r) : "f"(a), "f"(b), "f"(c));
  return r;
}
__device__ __forceinline__ void gp_barrier() { asm volatile("bar.sync 1, 256;" ::: "memory"); }   // the softmax threads

// 32 output columns of one row, times sigmoid(gate) where there is one
__device__ __forceinline__ void gp_store(const GroupedPrefillParams& p, __nv_bfloat16* orow, const __nv_bfloat16* grow, int col, float (&f)[32]) {
  const int n = p.s.vdim - col;
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    if (q * 8 >= n) break;
    if (grow != nullptr && p.s.head_gate) {
      const float a = gp_sigmoid(__bfloat162float(*grow));
#pragma unroll
      for (int i = 0; i < 8; ++i) f[q * 8 + i] *= a;
    } else if (grow != nullptr && p.gate_vec && q * 8 + 8 <= n) {
      const uint4 gv = *reinterpret_cast<const uint4*>(grow + col + q * 8);
      const uint32_t gg[4] = {gv.x, gv.y, gv.z, gv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 g2 = unpack_bf16x2(gg[i]);
        f[q * 8 + 2 * i] *= gp_sigmoid(g2.x);
        f[q * 8 + 2 * i + 1] *= gp_sigmoid(g2.y);
      }
    } else if (grow != nullptr) {
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (q * 8 + i < n) f[q * 8 + i] *= gp_sigmoid(__bfloat162float(grow[col + q * 8 + i]));
    }
    if (p.out_vec && q * 8 + 8 <= n) {
      *reinterpret_cast<uint4*>(orow + col + q * 8) =
          make_uint4(pack_bf16x2(f[q * 8], f[q * 8 + 1]), pack_bf16x2(f[q * 8 + 2], f[q * 8 + 3]),
                     pack_bf16x2(f[q * 8 + 4], f[q * 8 + 5]), pack_bf16x2(f[q * 8 + 6], f[q * 8 + 7]));
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (q * 8 + i < n) orow[col + q * 8 + i] = __float2bfloat16(f[q * 8 + i]);
    }
  }
}

template <int P, int MAPS, int SCORES>
__global__ void __launch_bounds__(GP_THREADS, 1)
grouped_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_kv, const GroupedPrefillParams p) {
  constexpr bool BIAS = SCORES == SCORES_BIAS, CAP = SCORES == SCORES_CAP, SLOPE = SCORES == SCORES_SLOPE;
  using L = GroupedPrefillSmem<P, BIAS>;
  extern __shared__ uint8_t gp_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(gp_raw) + 1023) & ~uintptr_t(1023));
  float* xch = reinterpret_cast<float*>(smem + L::OFF_X);
  float* lut = reinterpret_cast<float*>(smem + L::OFF_LUT);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR);
  uint64_t* q_full = bars;
  uint64_t *k_full = bars + 1, *k_empty = bars + 3;       // [2]: stage of the tile (one map) or map
  uint64_t *v_full = bars + 5, *v_empty = bars + 7;       // [2]
  uint64_t* s_full = bars + 9;                            // [2] per tile A / B
  uint64_t* p_full = bars + 11;                           // [2][2] per tile and half of the key tile (128 arrivals)
  uint64_t* o_full = bars + 15;                           // [2]
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + L::NUM_BARS);
  volatile uint32_t* abort_word = tmem_holder + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const GroupedShape& s = p.s;

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
    prefetch_tensormap(&tm_q);
    prefetch_tensormap(&tm_kv);
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, 512);
    tmem_relinquish();
  }
  pdl_sync();
  // Latest query tiles first (they may have more keys); the (portion, head) index varies fastest.
  const int bh = blockIdx.x % (p.portions * s.heads);
  const int blk = (int)(gridDim.x / (p.portions * s.heads)) - 1 - blockIdx.x / (p.portions * s.heads);
  const int b = bh / s.heads, h = bh - b * s.heads, g = h / (s.heads / s.kv_heads);
  const int row_base = p.cu[b], seq_len = p.cu[b + 1] - row_base;
  const int shift = seq_len > 0 ? p.positions[row_base] : 0;            // position of query 0
  const int last_pos = shift + seq_len - 1;
  // tile X covers queries [q0[X], q0[X] + 128) and walks the steps lo_t[X] .. n_kv_t[X] - 1; A's range starts and ends no later than
  // B's and the two leave no gap.  Step j is key tile j + (j < kept ? 0 : skip): with kept positions, B starts with them as A does.
  const int q0_t[2] = {MAPS == 1 ? blk * 256 : blk * 128, MAPS == 1 ? blk * 256 + 128 : blk * 128};
  int n_kv_t[2], lo_t[2];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    n_kv_t[x] = q0_t[x] < seq_len ? (min(q0_t[x] + 128, seq_len) + shift + 127) / 128 : 0;
    lo_t[x] = n_kv_t[x] > 0 ? max(0, first_seen(s, q0_t[x] + shift)) / 128 : 0;
  }
  const int kept = min((s.keep + 127) / 128, lo_t[0]), skip = kept > 0 ? lo_t[0] - kept : 0;
  if (s.keep > 0) {
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      n_kv_t[x] -= n_kv_t[x] > 0 ? skip : 0;
      lo_t[x] = 0;
    }
  }
  const int n_kv = max(n_kv_t[0], n_kv_t[1]), j0 = lo_t[0];
  auto key_tile = [&](int j) { return j < kept ? j : j + skip; };
  const bool active = n_kv > 0;
  if (BIAS && active) {
    const float* row = p.bias + (long long)h * p.bias_len;
    for (int i = threadIdx.x; i < p.bias_len + 2 * GP_LUT_PAD + 1; i += GP_THREADS)
      lut[i] = row[max(0, min(i - GP_LUT_PAD, p.bias_len - 1))] * 1.4426950408889634f;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;
  // columns: S_A [0,128)  S_B [128,256)  O_A [256,256+64P)  O_B [384,384+64P); P_X overlays the first 64 columns of S_X
  const int pd = (s.dim + 63) / 64, pv = (s.vdim + 63) / 64;            // panels that are loaded
  const int ksteps = (s.dim + 15) / 16;
  const int col_v = s.kv_heads * s.maps * s.kp + g * s.vp;

  if (warp == 0) {
    if (active) {
      const int pages = 128 / p.page_size;                              // per tile, at most 16
      const int last_page = last_pos / p.page_size;
      if (elect_one()) {
        mbar_expect_tx(q_full, (uint32_t)(2 * pd) * 16384u);
#pragma unroll
        for (int x = 0; x < 2; ++x)
          for (int pn = 0; pn < pd; ++pn)
            tma_load_2d(smem + L::OFF_Q + x * L::TILE + pn * 16384, &tm_q, q_full,
                        (h * MAPS + (MAPS == 2 ? x : 0)) * s.qp + pn * 64, row_base + q0_t[x]);
      }
      __syncwarp();
      for (int j = j0; j < n_kv; ++j) {
        const int i = j - j0;
        int page = 0;
        if (lane < pages) {
          const int pg = min(key_tile(j) * pages + lane, last_page);              // past the end: something valid
          page = pg < p.max_pages ? p.tables[(long long)b * p.max_pages + pg] : -1;
          if ((unsigned)page >= (unsigned)p.num_pages) {
            report_bad_arg(p.status, 19);
            page = 0;
          }
        }
        auto load = [&](uint8_t* dst, uint64_t* full, int col, int panels) {
          if (lane == 0) mbar_expect_tx(full, (uint32_t)panels * 16384u);
          __syncwarp();
          if (lane < pages)
            for (int pn = 0; pn < panels; ++pn)
              tma_load_2d(dst + pn * 16384 + lane * p.page_size * 128, &tm_kv, full, col + pn * 64, page * p.page_size);
          __syncwarp();
        };
        bool ok = true;
#pragma unroll
        for (int x = 0; x < MAPS; ++x) {
          const int st = MAPS == 1 ? (i & 1) : x;
          const uint32_t ph = MAPS == 1 ? ((i >> 1) & 1) : (i & 1);
          ok = __all_sync(0xffffffffu, ok && mbar_wait(&k_empty[st], ph ^ 1, abort_word));
          if (ok) load(smem + L::OFF_K + st * L::TILE, &k_full[st], (g * MAPS + x) * s.kp, pd);
        }
        ok = __all_sync(0xffffffffu, ok && mbar_wait(&v_empty[i & 1], ((i >> 1) & 1) ^ 1, abort_word));
        if (ok) load(smem + L::OFF_V + (i & 1) * L::TILE, &v_full[i & 1], col_v, pv);
        if (!ok) {
          *abort_word = ERR_WAIT_EMPTY;
          break;
        }
      }
    }
  } else if (warp == 1) {
    if (active && elect_one()) {
      constexpr uint32_t idesc_qk = make_idesc_bf16(128, 128, false, false);
      constexpr uint32_t idesc_pv = make_idesc_bf16(128, 64 * P, false, true);
      auto k_stage = [&](int x, int j) { return MAPS == 1 ? ((j - j0) & 1) : x; };
      auto k_phase = [&](int j) { return (uint32_t)(MAPS == 1 ? ((j - j0) >> 1) & 1 : (j - j0) & 1); };
      auto issue_s = [&](int x, int j) {   // S_X(j) = Q_X K_j^T
        const uint64_t q_desc = make_smem_desc(smem_u32(smem + L::OFF_Q + x * L::TILE), 16, 1024);
        const uint64_t k_desc = make_smem_desc(smem_u32(smem + L::OFF_K + k_stage(x, j) * L::TILE), 16, 1024);
#pragma unroll
        for (int k = 0; k < 4 * P; ++k) {
          if (k >= ksteps) break;
          const uint32_t off = ((k / 4) * 16384 + (k % 4) * 32) >> 4;
          umma_f16_ss(tmem_base + x * 128, q_desc + off, k_desc + off, idesc_qk, k > 0 ? 1u : 0u);
        }
        umma_commit(&s_full[x]);
        if (MAPS == 2) umma_commit(&k_empty[x]);
      };
      auto issue_pv = [&](int x, int j, int half) {   // O_X += P_X(j) V_j, half of the key tile at a time
        const uint64_t v_desc = make_smem_desc(smem_u32(smem + L::OFF_V + ((j - j0) & 1) * L::TILE), 16384, 1024);
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          const int k = half * 4 + kk;
          umma_f16_ts(tmem_base + 256 + x * 128, tmem_base + x * 128 + k * 8, v_desc + ((k * 2048) >> 4), idesc_pv,
                      (j > lo_t[x] || k > 0) ? 1u : 0u);
        }
        if (half == 1 && j == n_kv_t[x] - 1) umma_commit(&o_full[x]);
      };
      bool ok = mbar_wait(q_full, 0, abort_word) && mbar_wait(&k_full[0], 0, abort_word);
      if (ok) {
        tc_fence_after();
        if (n_kv_t[0] > 0) issue_s(0, j0);
        if (MAPS == 2) {
          ok = mbar_wait(&k_full[1], 0, abort_word);
          tc_fence_after();
          if (ok) issue_s(1, j0);
        } else {
          if (n_kv_t[1] > 0 && lo_t[1] == j0) issue_s(1, j0);
          umma_commit(&k_empty[0]);
        }
      }
      for (int j = j0; j < n_kv && ok; ++j) {
        const int st = (j - j0) & 1;
        const uint32_t ph = ((j - j0) >> 1) & 1;
        bool v_ready = false, k_ready = false;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          if (j >= lo_t[x] && j < n_kv_t[x]) {
            ok = mbar_wait(&p_full[2 * x], (j - lo_t[x]) & 1, abort_word) && (v_ready || mbar_wait(&v_full[st], ph, abort_word));
            if (!ok) break;
            v_ready = true;
            tc_fence_after();
            issue_pv(x, j, 0);
            ok = mbar_wait(&p_full[2 * x + 1], (j - lo_t[x]) & 1, abort_word);
            if (!ok) break;
            tc_fence_after();
            issue_pv(x, j, 1);
          }
          if (x == 1) umma_commit(&v_empty[st]);   // both tiles are done with V_j
          if (j + 1 >= lo_t[x] && j + 1 < n_kv_t[x]) {
            ok = (MAPS == 1 && k_ready) || mbar_wait(&k_full[k_stage(x, j + 1)], k_phase(j + 1), abort_word);
            if (!ok) break;
            k_ready = true;
            tc_fence_after();
            issue_s(x, j + 1);
          }
        }
        if (MAPS == 1 && ok && j + 1 < n_kv) umma_commit(&k_empty[st ^ 1]);   // both tiles are done with K_{j+1}
      }
      if (!ok) *abort_word = ERR_WAIT_FULL;
    }
  } else if (active) {
    // ----------------------------------------------------------------- softmax warps: one thread per query row
    const int x = (warp - 2) >> 2;              // tile A (warps 2-5) or B (warps 6-9)
    const int quarter = warp & 3;               // TMEM lanes [32*quarter, 32*quarter+32) are visible to this warp
    const int r = quarter * 32 + lane;          // row inside the query tile
    const int q0 = x == 0 ? q0_t[0] : q0_t[1];
    const int n_kv_x = x == 0 ? n_kv_t[0] : n_kv_t[1], lo_x = x == 0 ? lo_t[0] : lo_t[1];
    const int q_idx = q0 + r, q_key = q_idx + shift;      // query of this thread, its position
    const uint32_t lane_addr = uint32_t(quarter * 32) << 16;
    const uint32_t tm_s = tmem_base + x * 128 + lane_addr;
    const uint32_t tm_o = tmem_base + 256 + x * 128 + lane_addr;
    const float scale2 = BIAS ? 1.f : p.scale_log2;       // of what the second pass finds in tensor memory
    const float slope = CAP ? 2.f * p.scale_log2 / s.softcap : 0.f, top = s.softcap * LOG2E;      // see capped_log2
    const float part = slope / (2.f * LOG2E);             // a score's part of the cap
    float m_run = -INFINITY, l_run = 0.f;                 // running reference max in scaled log2 units, row sum relative to it
    bool ok = true;
    const __nv_bfloat16* grow = p.gate != nullptr && q_idx < seq_len ? p.gate + (long long)(row_base + q_idx) * p.ld_gate + gate_column(s, h) : nullptr;
    const int from = first_seen(s, q_key), from_last = first_seen(s, q0 + 127 + shift);     // of this row, of the tile's last one
    const float slope2 = SLOPE ? s.slopes[h] * LOG2E : 0.f;                                 // log2 units per token
    if (grow != nullptr && !s.head_gate)                                  // the epilogue's gate row into L2
      for (int i = 0; i < s.vdim; i += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(grow + i));
    for (int j = lo_x; j < n_kv_x; ++j) {
      if (!mbar_wait(&s_full[x], (j - lo_x) & 1, abort_word)) { ok = false; break; }
      tc_fence_after();
      const int k0 = key_tile(j) * 128;
      // tile touches the diagonal or the lower edge of the window (warp-uniform)
      const bool edge = (k0 + 127 > q0 + shift) || (k0 < from_last);
      const int kept_e = min(s.keep - k0, q_key - k0 + 1);      // keys k0 + e with e below are visible wherever the window is
      // Key k0 + e is visible iff e - first <= span as unsigned numbers (one comparison for both edges of the window).
      const int first = from - k0;
      const uint32_t span = (uint32_t)(q_key - from);
      const float base = SLOPE ? slope2 * (float)(k0 - q_key) : 0.f;      // of the tile's first key
      auto hidden = [&](int e) { return (uint32_t)(e - first) > span && e >= kept_e; };
      float mx = -INFINITY, mn = INFINITY;
      // pass 1: row maximum (plain: over the raw scores; BIAS: scores in log2 units with the bias, written back)
      const float* bp = nullptr;
      if (BIAS) {
        const bool far = q0 + shift - k0 - 127 >= p.bias_len - 1;       // the whole tile reads the last entry
        bp = lut + GP_LUT_PAD + (far ? p.bias_len - 1 + 127 + r : q_key - k0);
      }
      auto row_max = [&](const bool masked) __attribute__((always_inline)) {
        uint32_t sa[32], sb[32];
        tmem_ld_32x32(tm_s, sa);
        tmem_ld_wait();
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t (&cur)[32] = (c & 1) ? sb : sa;
          uint32_t (&nxt)[32] = (c & 1) ? sa : sb;
          if (c < 3) tmem_ld_32x32(tm_s + (c + 1) * 32, nxt);
          if (BIAS) {
#pragma unroll
            for (int i = 0; i < 32; ++i) cur[i] = __float_as_uint(fmaf(__uint_as_float(cur[i]), p.scale_log2, bp[-(c * 32 + i)]));
          }
          if (SLOPE) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              cur[i] = __float_as_uint(fmaf(__uint_as_float(cur[i]), p.scale_log2, fmaf(slope2, (float)(c * 32 + i), base)));
          }
          if (masked) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (hidden(c * 32 + i)) cur[i] = 0xff800000u;   // -inf
          }
#pragma unroll
          for (int i = 0; i < 32; i += 2) mx = gp_max3(mx, __uint_as_float(cur[i]), __uint_as_float(cur[i + 1]));
          if (CAP) {
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              const bool h0 = masked && hidden(c * 32 + i), h1 = masked && hidden(c * 32 + i + 1);
              mn = gp_min3(mn, h0 ? INFINITY : __uint_as_float(cur[i]), h1 ? INFINITY : __uint_as_float(cur[i + 1]));
            }
          }
          if (c < 3) tmem_ld_wait();
          if (BIAS) tmem_st_32x32(tm_s + c * 32, cur);
        }
        if (BIAS) tmem_st_wait();
      };
      if (edge) row_max(true);
      else row_max(false);
      const bool low = CAP && !__any_sync(0xffffffffu, fmaxf(mx, -mn) * part > 1.f);      // every score of the tile is below the cap
      if (CAP) mx = capped_log2(mx, slope, top);             // (no key: -cap, below or equal to what any key would give)
      else if (!BIAS && !SLOPE) mx *= p.scale_log2;
      // Lazy rescale: keep the old reference max unless it moved by more than 8 (a factor 256).
      float m_new = m_run;
      if (mx > m_run + 8.f) m_new = mx;
      const bool need = m_new != m_run;
      const float alpha = (m_run == -INFINITY) ? 0.f : gp_exp2(m_run - m_new);
      // S_X(j) was issued after P_X V_{j-1}, so that MMA has completed and O_X may be rescaled here.
      if (j > lo_x && __any_sync(0xffffffffu, need)) {
        const float f = need ? alpha : 1.f;
#pragma unroll 1
        for (int c = 0; c < 2 * P; ++c) {
          uint32_t o[32];
          tmem_ld_32x32(tm_o + c * 32, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
          tmem_st_32x32(tm_o + c * 32, o);
        }
      }
      if (k0 + 127 > last_pos) {       // value rows that this request has not written: zero, so that they cannot reach O even as 0 * NaN
        if (!mbar_wait(&v_full[(j - j0) & 1], ((j - j0) >> 1) & 1, abort_word)) { ok = false; break; }
        if (k0 + r > last_pos) {
          uint8_t* v = smem + L::OFF_V + ((j - j0) & 1) * L::TILE + r * 128;
#pragma unroll
          for (int pn = 0; pn < P; ++pn)
#pragma unroll
            for (int i = 0; i < 8; ++i) *reinterpret_cast<uint4*>(v + pn * 16384 + i * 16) = make_uint4(0, 0, 0, 0);
        }
        fence_proxy_async_smem();
      }
      // pass 2: P = exp2(S * scale - m), row sum, bf16 pack; P chunk c (16 packed columns) lands on S columns [16c, 16c+16), all of
      // which this thread has already read.  (A row whose window starts in a later tile has seen no key yet.)
      const float m_ref = m_new == -INFINITY ? 0.f : m_new;
      float sum = 0.f, sum1 = 0.f;
      auto weights = [&](const bool masked, const bool poly) __attribute__((always_inline)) {
        uint32_t sa[32], sb[32];
        tmem_ld_32x32(tm_s, sa);
        tmem_ld_wait();
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t (&sc)[32] = (c & 1) ? sb : sa;
          uint32_t (&nxt)[32] = (c & 1) ? sa : sb;
          uint32_t pk[16];
          if (c < 3) tmem_ld_32x32(tm_s + (c + 1) * 32, nxt);
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            float x0, x1;
            if (CAP && poly) {
              gp_tanh2(x0, x1, __uint_as_float(sc[i]), __uint_as_float(sc[i + 1]), part, top, m_ref);
            } else if (CAP) {
              x0 = gp_exp2(__uint_as_float(sc[i]) * slope);
              x1 = gp_exp2(__uint_as_float(sc[i + 1]) * slope);
              gp_fma2(x0, x1, gp_rcp(1.f + x0), gp_rcp(1.f + x1), -2.f * top, top - m_ref);
            } else if (SLOPE) {
              const float2 d = __ffma2_rn(make_float2(slope2, slope2), make_float2((float)(c * 32 + i), (float)(c * 32 + i + 1)),
                                          make_float2(base - m_ref, base - m_ref));
              const float2 y = __ffma2_rn(make_float2(__uint_as_float(sc[i]), __uint_as_float(sc[i + 1])), make_float2(scale2, scale2), d);
              x0 = y.x;
              x1 = y.y;
            } else {
              gp_fma2(x0, x1, __uint_as_float(sc[i]), __uint_as_float(sc[i + 1]), scale2, -m_ref);
            }
            float e0 = gp_exp2(x0), e1 = gp_exp2(x1);
            if (!BIAS && masked) {                       // (BIAS: hidden keys are -inf already)
              e0 = hidden(c * 32 + i) ? 0.f : e0;
              e1 = hidden(c * 32 + i + 1) ? 0.f : e1;
            }
            gp_add2(sum, sum1, e0, e1);
            pk[i / 2] = pack_bf16x2(e0, e1);
          }
          if (c < 3) tmem_ld_wait();   // before the store below: wait::ld covers the prefetched chunk
          tmem_st_32x16(tm_s + c * 16, pk);
          if (c == 1 || c == 3) {      // publish this half of P
            tmem_st_wait();
            tc_fence_before();
            mbar_arrive(&p_full[2 * x + (c >> 1)]);
          }
        }
      };
      if (CAP && low) {
        if (edge) weights(true, true);
        else weights(false, true);
      } else {
        if (!BIAS && edge) weights(true, false);
        else weights(false, false);
      }
      l_run = l_run * (need ? alpha : 1.f) + (sum + sum1);
      m_run = m_new;
    }
    // ------------------------------------------------------------------- epilogue
    const bool valid = q_idx < seq_len;
    __nv_bfloat16* orow = p.o + (long long)(row_base + (valid ? q_idx : 0)) * p.ld_o + h * s.vdim;
    if (MAPS == 1) {
      if (ok && n_kv_x > 0) ok = mbar_wait(&o_full[x], 0, abort_word);
      if (ok && n_kv_x > 0) {
        tc_fence_after();
        if (s.sink != nullptr) l_run += gp_exp2(fminf(fmaf(s.sink[h], LOG2E, -m_run), 126.f));
        const float inv_l = 1.f / l_run;
#pragma unroll 1
        for (int c = 0; c < 2 * P; ++c) {
          uint32_t o[32];
          tmem_ld_32x32(tm_o + c * 32, o);
          tmem_ld_wait();
          if (valid && c * 32 < s.vdim) {
            float f[32];
#pragma unroll
            for (int i = 0; i < 32; ++i) f[i] = __uint_as_float(o[i]) * inv_l;
            gp_store(p, orow, grow, c * 32, f);
          }
        }
      }
    } else {
      // both maps of this query row; the two threads of a row take half of the columns each
      xch[x * 128 + r] = 1.f / l_run;
      if (ok) ok = mbar_wait(&o_full[0], 0, abort_word) && mbar_wait(&o_full[1], 0, abort_word);
      tc_fence_after();
      gp_barrier();
      const float f1 = xch[r], f2 = xch[128 + r] * s.difference;
      float o[P][32], ss = 0.f;
#pragma unroll
      for (int c = 0; c < P; ++c) {
        uint32_t a[32], d[32];
        const int col = (x * P + c) * 32;
        tmem_ld_32x32(tmem_base + 256 + lane_addr + col, a);
        tmem_ld_32x32(tmem_base + 384 + lane_addr + col, d);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          o[c][i] = __uint_as_float(a[i]) * f1 - __uint_as_float(d[i]) * f2;
          if (col + i < s.vdim) ss = fmaf(o[c][i], o[c][i], ss);
        }
      }
      xch[256 + x * 128 + r] = ss;
      gp_barrier();
      const float inv = rsqrtf((xch[256 + r] + xch[384 + r]) / (float)s.vdim + s.eps) * s.out_scale;
      if (valid && ok) {
#pragma unroll
        for (int c = 0; c < P; ++c) {
          const int col = (x * P + c) * 32;
          if (col >= s.vdim) break;
#pragma unroll
          for (int i = 0; i < 32; ++i) o[c][i] *= inv;
          gp_store(p, orow, grow, col, o[c]);
        }
      }
    }
    if (!ok && lane == 0) *abort_word = ERR_WAIT_TMEM_FULL;
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

template <int P, int MAPS, int SCORES>
static int launch_grouped_prefill(const CUtensorMap& tm_q, const CUtensorMap& tm_kv, const GroupedPrefillParams& p, cudaStream_t st) {
  const int smem = GroupedPrefillSmem<P, SCORES == SCORES_BIAS>::total(p.bias_len);
  auto kern = grouped_prefill_kernel<P, MAPS, SCORES>;
  static int configured = 0;
  if (smem > configured) {
    if (smem > 232448 || cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
    configured = smem;
  }
  const long long grid = (long long)p.portions * p.s.heads * (MAPS == 1 ? (p.n_qblk + 1) / 2 : p.n_qblk);
  if (grid > 0x7fffffffll) return -13;
  launch_dep(kern, (unsigned)grid, GP_THREADS, smem, st, tm_q, tm_kv, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace b200

using namespace b200;

// q: (total_q, heads * maps * qp) with qp a multiple of 64, portion b in rows cu[b] .. cu[b + 1] - 1 (at most max_q of them), its first
// query at position positions[cu[b]]; line b of the tables holds its pages.  dim and vdim up to 128, page_size a divisor of 128 of
// at least 8, a softcap only for one map and without a bias, scale positive unless there is a bias, bias_len at most B200_GROUPED_BIAS_MAX.
constexpr int B200_GROUPED_BIAS_MAX = 6000;

extern "C" int b200_grouped_prefill(const void* q, const void* cache, void* o, long long ld_o, const void* gate, long long ld_gate,
                                    const float* bias, int bias_len, const int* cu, const int* positions, const int* tables,
                                    int portions, int max_q, int total_q, int max_pages, int page_size, int num_pages,
                                    const GroupedShape* s, uint32_t* status, cudaStream_t st) {
  if (portions <= 0 || total_q <= 0) return 0;
  if (!shape_ok(*s) || s->dim > 128 || s->vdim > 128 || s->qp % 64 || page_size < 8 || 128 % page_size || max_q <= 0) return -10;
  if (bias != nullptr ? (bias_len <= 0 || bias_len > B200_GROUPED_BIAS_MAX) : !(s->scale > 0.f)) return -11;
  if (s->softcap > 0.f && (bias != nullptr || s->maps != 1)) return -12;
  if (s->slopes != nullptr && bias != nullptr) return -12;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15) return -10;
  const uint64_t qw = (uint64_t)s->heads * s->maps * s->qp, width = (uint64_t)s->kv_heads * (s->maps * s->kp + s->vp);
  CUtensorMap tm_q, tm_kv;
  if (make_tmap_bf16_2d(&tm_q, q, (uint64_t)total_q, qw, qw, 64, 128)) return -20;
  if (make_tmap_bf16_2d(&tm_kv, cache, (uint64_t)num_pages * page_size, width, width, 64, (uint32_t)page_size)) return -21;
  GroupedPrefillParams p;
  p.o = (__nv_bfloat16*)o; p.gate = (const __nv_bfloat16*)gate; p.ld_o = ld_o; p.ld_gate = ld_gate; p.bias = bias;
  p.bias_len = bias != nullptr ? bias_len : 0; p.cu = cu; p.positions = positions; p.tables = tables; p.portions = portions;
  p.n_qblk = (max_q + 127) / 128; p.max_pages = max_pages; p.page_size = page_size; p.num_pages = num_pages; p.s = *s;
  p.scale_log2 = s->scale * 1.4426950408889634f; p.status = status;
  p.out_vec = s->vdim % 8 == 0 && ld_o % 8 == 0 && (reinterpret_cast<uintptr_t>(o) & 15) == 0;
  p.gate_vec = s->vdim % 8 == 0 && ld_gate % 8 == 0 && (reinterpret_cast<uintptr_t>(gate) & 15) == 0;
  const bool wide = s->dim > 64 || s->vdim > 64;
#define GROUPED_PREFILL(MAPS, SCORES)                                          \
  return wide ? launch_grouped_prefill<2, MAPS, SCORES>(tm_q, tm_kv, p, st)    \
              : launch_grouped_prefill<1, MAPS, SCORES>(tm_q, tm_kv, p, st)
  if (s->maps == 1) {
    if (bias != nullptr) GROUPED_PREFILL(1, SCORES_BIAS);
    if (s->slopes != nullptr) GROUPED_PREFILL(1, SCORES_SLOPE);
    if (s->softcap > 0.f) GROUPED_PREFILL(1, SCORES_CAP);
    GROUPED_PREFILL(1, SCORES_PLAIN);
  }
  if (bias != nullptr) GROUPED_PREFILL(2, SCORES_BIAS);
  GROUPED_PREFILL(2, SCORES_PLAIN);
#undef GROUPED_PREFILL
}
