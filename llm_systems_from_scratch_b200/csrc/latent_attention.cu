// Latent attention over a paged cache of latents.  Keys and values of all heads are linear images of one cached vector c
// per token (k_h = W_uk,h c, v_h = W_uv,h c), so a query is moved into latent space first (q'_h = W_uk,h^T q_h, a small
// GEMM per head): score = q'_h . c * scale, and sum_j p_j c_j goes through W_uv,h afterwards.  Every cached byte is then
// read once for all heads.  The mask is a sliding window: position i sees the `window` positions up to and including i.
//
// A rotated key part shared by all heads may follow the latent: the score gains q_rot,h . k_rot, so a query in latent space is
// [q'_h, q_rot,h], a cached vector [c, k_rot], and only c is summed up.
//
// Cache layout per layer run: (num_pages, page_size, width), width = vwidth + rotated part, each rounded up to 8 elements, zero padded
// (vwidth: the latent).
#include "typed.cuh"

namespace b200 {

// Row-wise norms of the two latents of a layer and the append to the cache:
//   cq[row] = rms_norm(proj[row, 0 : q_rank]) * wq,   cache[slot[row]] = rms_norm(proj[row, q_rank : q_rank + kv_rank]) * wkv
// One warp per row; the row is read twice (the second read hits L1).
template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_norm_append_kernel(
    const T* __restrict__ proj, long long ld_proj, const T* __restrict__ wq, const T* __restrict__ wkv, T* __restrict__ cq,
    long long ld_cq, T* __restrict__ cache, const long long* __restrict__ slots, int rows, int q_rank, int kv_rank, int width,
    long long num_slots, float eps, uint32_t* __restrict__ status) {
  pdl_sync();
  const int lane = threadIdx.x & 31;
  const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (row >= rows) return;
  const T* pr = proj + (long long)row * ld_proj;
  const T* pk = pr + q_rank;
  float sq = 0.f, skv = 0.f;
#pragma unroll 4
  for (int c = lane * VEC; c < q_rank; c += 32 * VEC) {
    float f[VEC];
    load_vec<VEC>(pr + c, f);
#pragma unroll
    for (int i = 0; i < VEC; ++i) sq += f[i] * f[i];
  }
#pragma unroll 4
  for (int c = lane * VEC; c < kv_rank; c += 32 * VEC) {
    float f[VEC];
    load_vec<VEC>(pk + c, f);
#pragma unroll
    for (int i = 0; i < VEC; ++i) skv += f[i] * f[i];
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    skv += __shfl_xor_sync(0xffffffffu, skv, o);
  }
  const float rq = rsqrtf(sq / (float)q_rank + eps), rkv = rsqrtf(skv / (float)kv_rank + eps);
  T* q = cq + (long long)row * ld_cq;
#pragma unroll 4
  for (int c = lane * VEC; c < q_rank; c += 32 * VEC) {
    float f[VEC], g[VEC];
    load_vec<VEC>(pr + c, f);
    load_vec<VEC>(wq + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) f[i] = f[i] * rq * g[i];
    store_vec<VEC>(q + c, f);
  }
  const long long slot = slots[row];
  if (slot < 0) return;                       // padding row of the batch
  if (slot >= num_slots) {
    if (lane == 0) report_bad_arg(status, 4);
    return;
  }
  T* dst = cache + slot * width;
#pragma unroll 4
  for (int c = lane * VEC; c < kv_rank; c += 32 * VEC) {
    float f[VEC], g[VEC];
    load_vec<VEC>(pk + c, f);
    load_vec<VEC>(wkv + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) f[i] = f[i] * rkv * g[i];
    store_vec<VEC>(dst + c, f);
  }
}

// Rotation of interleaved pairs (elements 2i and 2i + 1) and append.  One block per row: warp 0 norms the latent and rotates the key
// part on their way to the cache, the other warps rotate the heads' query parts: for the first `absorbed` rows behind the queries in
// latent space, for the others in place.
struct LatentRotateParams {
  void* q;                     // (rows, ld_q)
  const void* kv;              // (rows, ld_kv)
  long long ld_q, ld_kv;
  int q_col, q_pitch;          // rotated part of head h: columns q_col + h * q_pitch ... of q
  int kv_col;                  // the latent's first column of kv, negative: no latent here
  int k_col;                   // the key part's first column of kv, negative: none
  const void* wkv;
  void* ql;                    // (absorbed, heads * width)
  void* cache;
  const float* cos_sin;        // (2, ctx, rot / 2)
  const int* positions;
  const long long* slots;
  int rows, absorbed, heads, kv_rank, vwidth, width, rot, ctx;
  long long num_slots;
  float eps;
  uint32_t* status;
};

// VEC elements (whole pairs) of a rotated vector: src -> dst
template <typename T, int VEC>
__device__ __forceinline__ void rotate_pairs(const T* src, T* dst, const float* cs, const float* sn) {
  if constexpr (VEC == 8) {                   // bf16, 16 bytes
    const uint4 raw = *reinterpret_cast<const uint4*>(src);
    const float4 c = *reinterpret_cast<const float4*>(cs), s = *reinterpret_cast<const float4*>(sn);
    const uint32_t in[4] = {raw.x, raw.y, raw.z, raw.w};
    const float cc[4] = {c.x, c.y, c.z, c.w}, ss[4] = {s.x, s.y, s.z, s.w};
    uint32_t out[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 v = unpack_bf16x2(in[i]);
      out[i] = pack_bf16x2(v.x * cc[i] - v.y * ss[i], v.y * cc[i] + v.x * ss[i]);
    }
    *reinterpret_cast<uint4*>(dst) = make_uint4(out[0], out[1], out[2], out[3]);
    return;
  }
  float f[VEC];
  if constexpr (VEC == 4) {
    load_vec<4>(src, f);
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) f[i] = to_f(src[i]);
  }
#pragma unroll
  for (int i = 0; i < VEC; i += 2) {
    const float c = cs[i / 2], s = sn[i / 2], u = f[i], v = f[i + 1];
    f[i] = u * c - v * s;
    f[i + 1] = v * c + u * s;
  }
  if constexpr (VEC == 4) {
    store_vec<4>(dst, f);
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) from_f(dst[i], f[i]);
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_rotate_kernel(const LatentRotateParams p) {
  pdl_sync();
  const int row = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  T* pr = reinterpret_cast<T*>(p.q) + (long long)row * p.ld_q;
  const T* kr = reinterpret_cast<const T*>(p.kv) + (long long)row * p.ld_kv;
  int pos = p.positions[row];
  if (pos < 0 || pos >= p.ctx) {
    if (threadIdx.x == 0) report_bad_arg(p.status, 21);
    pos = 0;
  }
  const int half = p.rot / 2;
  const float* cs = p.cos_sin + (long long)pos * half;
  const float* sn = cs + (long long)p.ctx * half;
  if (warp > 0) {
    const int per = p.rot / VEC, total = p.heads * per;
    for (int i = threadIdx.x - 32; i < total; i += blockDim.x - 32) {
      const int h = i / per, c = (i - h * per) * VEC;
      T* src = pr + p.q_col + h * p.q_pitch + c;
      T* dst = row < p.absorbed ? reinterpret_cast<T*>(p.ql) + ((long long)row * p.heads + h) * p.width + p.vwidth + c : src;
      rotate_pairs<T, VEC>(src, dst, cs + c / 2, sn + c / 2);
    }
    const int pad = p.width - p.vwidth - p.rot;
    if (row < p.absorbed)
      for (int i = threadIdx.x - 32; i < p.heads * pad; i += blockDim.x - 32)
        from_f(reinterpret_cast<T*>(p.ql)[((long long)row * p.heads + i / pad) * p.width + p.vwidth + p.rot + i % pad], 0.f);
    return;
  }
  const long long slot = p.slots[row];
  if (slot < 0) return;                       // padding row of the batch
  if (slot >= p.num_slots) {
    if (lane == 0) report_bad_arg(p.status, 22);
    return;
  }
  T* dst = reinterpret_cast<T*>(p.cache) + slot * p.width;
  if (p.k_col >= 0) {
    for (int c = lane * VEC; c < p.rot; c += 32 * VEC) rotate_pairs<T, VEC>(kr + p.k_col + c, dst + p.vwidth + c, cs + c / 2, sn + c / 2);
    for (int c = p.vwidth + p.rot + lane; c < p.width; c += 32) from_f(dst[c], 0.f);
  }
  if (p.kv_col < 0) return;
  constexpr int LV = VEC >= 4 ? 4 : 1;
  const T* src = kr + p.kv_col;
  float ss = 0.f;
#pragma unroll 4
  for (int c = lane * LV; c < p.kv_rank; c += 32 * LV) {
    float f[LV];
    load_vec<LV>(src + c, f);
#pragma unroll
    for (int i = 0; i < LV; ++i) ss += f[i] * f[i];
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float r = rsqrtf(ss / (float)p.kv_rank + p.eps);
#pragma unroll 4
  for (int c = lane * LV; c < p.kv_rank; c += 32 * LV) {
    float f[LV], g[LV];
    load_vec<LV>(src + c, f);
    load_vec<LV>(reinterpret_cast<const T*>(p.wkv) + c, g);
#pragma unroll
    for (int i = 0; i < LV; ++i) f[i] = f[i] * r * g[i];
    store_vec<LV>(dst + c, f);
  }
  for (int c = p.kv_rank + lane; c < p.vwidth; c += 32) from_f(dst[c], 0.f);
}

// Latents of the keys that the portions of a step can see, packed for the prefill kernel:
//   out[cu_k[b] + i] = latent of position first_k[b] + i of portion b
template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(
    const T* __restrict__ cache, T* __restrict__ out, const int* __restrict__ cu_k, const int* __restrict__ first_k,
    const int* __restrict__ tables, int portions, int max_pages, int page_size, int num_pages, int width, int vec_per_row,
    uint32_t* __restrict__ status) {
  pdl_sync();
  const int total = cu_k[portions];
  const int lanes = vec_per_row;               // 16-byte vectors of a row
  const long long n = (long long)total * lanes;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const int row = (int)(i / lanes), v = (int)(i - (long long)row * lanes);
    int lo = 0, hi = portions - 1;             // last portion whose first row is <= row
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (cu_k[mid] <= row) lo = mid; else hi = mid - 1;
    }
    const int pos = first_k[lo] + row - cu_k[lo];
    const int pg = pos / page_size;
    int page = (pos >= 0 && pg < max_pages) ? tables[(long long)lo * max_pages + pg] : -1;
    uint4 val = make_uint4(0, 0, 0, 0);
    if ((unsigned)page < (unsigned)num_pages)
      val = reinterpret_cast<const uint4*>(cache + ((long long)page * page_size + pos % page_size) * width)[v];
    else
      report_bad_arg(status, 5);
    reinterpret_cast<uint4*>(out + (long long)row * width)[v] = val;
  }
}

// General form, any head count, any width, T = bf16 or fp32: one warp per (row, head), keys one after the other.
// q: (rows, heads * width), o: (rows, heads * vwidth).  row_seq[row] names the row's line of `tables`.
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_rows_kernel(
    const T* __restrict__ q, const T* __restrict__ cache, T* __restrict__ o, const int* __restrict__ row_seq,
    const int* __restrict__ positions, const long long* __restrict__ slots, const int* __restrict__ tables, int seqs,
    int rows, int heads, int width, int vwidth, int max_pages, int page_size, int num_pages, int window, float scale,
    uint32_t* __restrict__ status) {
  pdl_sync();
  extern __shared__ float lsm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + warp;
  if (item >= (long long)rows * heads) return;
  const int row = (int)(item / heads), h = (int)(item - (long long)row * heads);
  float* qs = lsm + warp * 2 * width;
  float* acc = qs + width;
  const T* qr = q + ((long long)row * heads + h) * width;
  T* orow = o + ((long long)row * heads + h) * vwidth;
  for (int c = lane; c < width; c += 32) { qs[c] = to_f(qr[c]) * scale; acc[c] = 0.f; }
  float m = -INFINITY, l = 0.f;
  const int seq = row_seq != nullptr ? row_seq[row] : row;
  const bool live = slots[row] >= 0 && seq >= 0 && seq < seqs;
  const int pos = positions[row];
  if (live) {
    const int* table = tables + (long long)seq * max_pages;
    const int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
    for (int j = lo; j <= pos; ++j) {
      const int pg = j / page_size;
      const int page = pg < max_pages ? table[pg] : -1;
      if ((unsigned)page >= (unsigned)num_pages) {
        if (lane == 0) report_bad_arg(status, 6);
        break;
      }
      const T* c = cache + ((long long)page * page_size + j % page_size) * width;
      float s = 0.f;
      for (int i = lane; i < width; i += 32) s = fmaf(qs[i], to_f(c[i]), s);
#pragma unroll
      for (int k = 16; k > 0; k >>= 1) s += __shfl_xor_sync(0xffffffffu, s, k);
      const float mn = fmaxf(m, s);
      const float a = expf(m - mn), e = expf(s - mn);      // first key: exp(-inf) = 0
      l = l * a + e;
      for (int i = lane; i < vwidth; i += 32) acc[i] = acc[i] * a + e * to_f(c[i]);
      m = mn;
    }
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int c = lane; c < vwidth; c += 32) from_f(orow[c], acc[c] * inv);
}

// ------------------------------------------------------------------------------- decode, bf16, on the tensor cores
// One CTA = one row (request), up to 16 * HG of its heads and one split of the window.  All heads share the cached latents,
// so the score and value products are (heads x width) by (width x tokens) and back: with 16 heads that is ~32 FLOP per
// cached byte, too much for the FMA pipes but little for mma.sync at M = 16, and the kernel stays bound by reading the
// cache.  Tiles of 32 tokens are copied by cp.async into a three-stage ring straight from the pages; the eight warps of a
// group of 16 heads compute 8 tokens' scores over half of the latent columns each (the softmax adds the halves), then own
// an eighth of the latent columns of the output: many short chains of MMAs instead of few long ones.  The queries
// stay in registers as MMA fragments, the page of a tile's tokens is looked up a tile earlier than its copy is issued, and
// the softmax is online, in fp32.
constexpr int LD_BT = 32;       // tokens per tile
constexpr int LD_STAGES = 3;

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}

struct LatentDecodeParams {
  const __nv_bfloat16* q;       // (rows, heads * width)
  const __nv_bfloat16* cache;
  __nv_bfloat16* o;             // (rows, heads * vwidth)
  float* part_o;                // (rows, heads, splits, vwidth) when splits > 1
  float* part_ml;               // (rows, heads, splits, 2)
  const int* positions;
  const long long* slots;
  const int* tables;            // line i for row i
  int rows, heads, width, vwidth, max_pages, page_size, num_pages, window, splits;
  float scale_log2;
  uint32_t* status;
};

template <int KT>
struct LatentDecodeSmem {
  static constexpr int KP = KT * 64;            // columns of a cached vector, padded
  static constexpr int PITCH = KP + 8;          // an odd number of 16-byte pieces: ldmatrix without bank conflicts
  static constexpr int bytes(int hg) {
    return LD_STAGES * LD_BT * PITCH * 2 + hg * 16 * (2 * (LD_BT + 4) * 4 + (LD_BT + 8) * 2 + 8);
  }
};

// KT, NT: 64-column pieces of a cached vector and of the part of it that is summed up
template <int KT, int NT, int HG>
__global__ void __launch_bounds__(256 * HG, HG == 1 && KT <= 8 ? 2 : 1) latent_decode_kernel(const LatentDecodeParams p) {
  using L = LatentDecodeSmem<KT>;
  constexpr int KP = L::KP, PITCH = L::PITCH, M = HG * 16, SP = LD_BT + 4, PP = LD_BT + 8, THREADS = 256 * HG;
  constexpr int ROWS = LD_BT / (8 * HG);                                    // token rows a warp copies per tile
  extern __shared__ __align__(16) uint8_t ld_smem[];
  __nv_bfloat16* sc = reinterpret_cast<__nv_bfloat16*>(ld_smem);            // [LD_STAGES][LD_BT][PITCH]
  float* ss = reinterpret_cast<float*>(sc + LD_STAGES * LD_BT * PITCH);     // [2][M][SP]
  __nv_bfloat16* sp = reinterpret_cast<__nv_bfloat16*>(ss + 2 * M * SP);        // [M][PP]
  float* salpha = reinterpret_cast<float*>(sp + M * PP);                    // [M]
  float* sl = salpha + M;                                                   // [M]
  pdl_sync();
  const int row = blockIdx.x, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int grp = warp >> 3, wq = warp & 7;                                 // group of 16 heads, warp inside it
  const int tq = wq & 3, kh = wq >> 2;                                      // its 8 tokens, its half of the columns
  const int h0 = blockIdx.y * M;
  const int pos = p.positions[row];
  const bool live = p.slots[row] >= 0 && pos >= 0;
  const int lo = (p.window > 0 && pos - p.window + 1 > 0) ? pos - p.window + 1 : 0;
  const int n = live ? pos - lo + 1 : 0;
  const int per = ((n + p.splits - 1) / p.splits + LD_BT - 1) / LD_BT * LD_BT;
  const int t0 = lo + split * per;
  const int t1 = min(lo + n, t0 + per);
  const int tiles = t1 > t0 ? (t1 - t0 + LD_BT - 1) / LD_BT : 0;
  const int vecs = p.width / 8;                                             // 16-byte pieces of a latent
  const int* table = p.tables + (long long)row * p.max_pages;

  // cache row of token (warp * ROWS + lane) of a tile, looked up by the first ROWS lanes; -1 = past the end
  auto look_up = [&](int tile) -> long long {
    const int t = t0 + tile * LD_BT + warp * ROWS + (lane & (ROWS - 1));
    if (t >= t1) return -1;
    const int pg = t / p.page_size;
    const int page = pg < p.max_pages ? table[pg] : -1;
    if ((unsigned)page < (unsigned)p.num_pages) return (long long)page * p.page_size + t % p.page_size;
    report_bad_arg(p.status, 9);
    return -1;
  };
  auto request = [&](int tile, long long src) {
    __nv_bfloat16* dst = sc + (tile % LD_STAGES) * LD_BT * PITCH;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      const long long s = __shfl_sync(0xffffffffu, src, r);
      __nv_bfloat16* d = dst + (warp * ROWS + r) * PITCH;
      for (int v = lane; v < vecs; v += 32) {
        if (s >= 0) cp_async16(smem_u32(d + v * 8), p.cache + s * p.width + v * 8);
        else *reinterpret_cast<uint4*>(d + v * 8) = make_uint4(0, 0, 0, 0);  // finite; masked below
      }
    }
  };
  auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };

  if (p.width < KP) {                                                       // pad columns of the ring stay zero
    for (int i = threadIdx.x; i < LD_STAGES * LD_BT * (KP / 8 - vecs); i += THREADS) {
      const int r = i / (KP / 8 - vecs), v = vecs + i - r * (KP / 8 - vecs);
      *reinterpret_cast<uint4*>(sc + r * PITCH + v * 8) = make_uint4(0, 0, 0, 0);
    }
  }
  // The queries pass through the ring's last stage, which no tile uses before the first iteration.
  {
    __nv_bfloat16* sq = sc + (LD_STAGES - 1) * LD_BT * PITCH;               // [M][PITCH], M <= LD_BT
    const int q_rows = min(M, p.heads - h0);
    for (int i = threadIdx.x; i < q_rows * vecs; i += THREADS) {
      const int r = i / vecs, v = i - r * vecs;
      cp_async16(smem_u32(sq + r * PITCH + v * 8), p.q + ((long long)row * p.heads + h0 + r) * p.width + v * 8);
    }
    commit();
  }
#pragma unroll
  for (int i = 0; i < LD_STAGES - 1; ++i) {                                 // one group per tile, empty ones included
    if (i < tiles) request(i, look_up(i));
    commit();
  }
  long long next_src = LD_STAGES - 1 < tiles ? look_up(LD_STAGES - 1) : -1;
  asm volatile("cp.async.wait_group %0;" ::"n"(LD_STAGES - 1) : "memory");  // the queries have landed
  __syncthreads();
  uint32_t qf[KT * 2][4];                  // A fragments of this group's 16 heads, this warp's half of the columns
  {
    const uint32_t a_addr = smem_u32(sc + ((LD_STAGES - 1) * LD_BT + grp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PITCH +
                                     kh * KT * 32 + (lane >> 4) * 8);
#pragma unroll
    for (int k = 0; k < KT * 2; ++k) ldsm_x4(qf[k], a_addr + k * 32);
  }
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
  const int sr = grp * 16 + ((threadIdx.x & 255) >> 4), se = (threadIdx.x & 15) * 2;  // softmax: row, first of two columns
  float m_run = -INFINITY, l_run = 0.f;                                     // of row sr, the same in its 16 threads

  for (int it = 0; it < tiles; ++it) {
    asm volatile("cp.async.wait_group %0;" ::"n"(LD_STAGES - 2) : "memory");
    __syncthreads();                       // tile `it` is in shared memory, everybody is done with tile it - 1
    if (it + LD_STAGES - 1 < tiles) {
      request(it + LD_STAGES - 1, next_src);
      next_src = it + LD_STAGES < tiles ? look_up(it + LD_STAGES) : -1;
    }
    commit();
    const __nv_bfloat16* c = sc + (it % LD_STAGES) * LD_BT * PITCH;
    // ---- scores of 8 tokens for the group's heads
    float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
    const uint32_t b_addr = smem_u32(c + (tq * 8 + (lane & 7)) * PITCH + kh * KT * 32 + (lane >> 3) * 8);
#pragma unroll
    for (int k = 0; k < KT; ++k) {
      uint32_t b[4];
      ldsm_x4(b, b_addr + k * 64);
      mma_bf16(s0, qf[2 * k], b[0], b[1]);
      mma_bf16(s1, qf[2 * k + 1], b[2], b[3]);
    }
    {
      const int r = kh * M + grp * 16 + (lane >> 2), col = tq * 8 + (lane & 3) * 2;
      const int tok = t0 + it * LD_BT + col;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float v = (s0[i] + s1[i]) * p.scale_log2;
        ss[(r + (i >> 1) * 8) * SP + col + (i & 1)] = (tok + (i & 1) < t1) ? v : -INFINITY;
      }
    }
    __syncthreads();
    // ---- online softmax: sixteen threads per head row
    {
      const float2 va = *reinterpret_cast<const float2*>(ss + sr * SP + se);
      const float2 vb = *reinterpret_cast<const float2*>(ss + (M + sr) * SP + se);
      const float x = va.x + vb.x, y = va.y + vb.y;
      float mx = fmaxf(x, y);
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float mn = fmaxf(m_run, mx);               // finite: every tile holds at least one token
      const float p0 = exp2f(x - mn), p1 = exp2f(y - mn);
      float sum = p0 + p1;
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      const float alpha = exp2f(m_run - mn);
      l_run = l_run * alpha + sum;
      m_run = mn;
      *reinterpret_cast<uint32_t*>(sp + sr * PP + se) = pack_bf16x2(p0, p1);
      if ((threadIdx.x & 15) == 0) salpha[sr] = alpha;
    }
    __syncthreads();
    // ---- O = alpha O + P C for this warp's eighth of the columns
    const uint32_t v_addr = smem_u32(c + ((lane & 7) + ((lane >> 3) & 1) * 8) * PITCH + wq * (NT * 8) + (lane >> 4) * 8);
    const uint32_t p_addr = smem_u32(sp + (grp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PP + (lane >> 4) * 8);
    const float a0 = salpha[grp * 16 + (lane >> 2)], a1 = salpha[grp * 16 + (lane >> 2) + 8];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      acc[j][0] *= a0; acc[j][1] *= a0; acc[j][2] *= a1; acc[j][3] *= a1;
    }
#pragma unroll
    for (int k = 0; k < LD_BT / 16; ++k) {
      uint32_t a[4];
      ldsm_x4(a, p_addr + k * 32);
#pragma unroll
      for (int j = 0; j < NT / 2; ++j) {
        uint32_t b[4];
        ldsm_x4_t(b, v_addr + k * 16 * PITCH * 2 + j * 32);
        mma_bf16(acc[2 * j], a, b[0], b[1]);
        mma_bf16(acc[2 * j + 1], a, b[2], b[3]);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  // ---- results: normalised here, or left as (max, sum, unnormalised output) for the merge
  if ((threadIdx.x & 15) == 0) {
    sl[sr] = l_run;
    if (p.splits > 1 && h0 + sr < p.heads) {
      float* ml = p.part_ml + (((long long)row * p.heads + h0 + sr) * p.splits + split) * 2;
      ml[0] = m_run;
      ml[1] = l_run;
    }
  }
  __syncthreads();
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int r = grp * 16 + (lane >> 2) + half * 8;
    if (h0 + r >= p.heads) continue;
    const float inv = sl[r] > 0.f ? 1.f / sl[r] : 0.f;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int col = wq * (NT * 8) + j * 8 + (lane & 3) * 2;
      if (col >= p.vwidth) continue;
      const float x = acc[j][half * 2], y = acc[j][half * 2 + 1];
      if (p.splits > 1)
        *reinterpret_cast<float2*>(p.part_o + (((long long)row * p.heads + h0 + r) * p.splits + split) * p.vwidth + col) =
            make_float2(x, y);
      else
        *reinterpret_cast<uint32_t*>(p.o + ((long long)row * p.heads + h0 + r) * p.vwidth + col) = pack_bf16x2(x * inv, y * inv);
    }
  }
}

__global__ void __launch_bounds__(128) latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                           __nv_bfloat16* __restrict__ o, int splits, int width) {
  pdl_sync();
  const long long base = (long long)blockIdx.x * splits;          // (row, head)
  float gm = -INFINITY;
  for (int s = 0; s < splits; ++s) gm = fmaxf(gm, part_ml[(base + s) * 2]);
  float gl = 0.f;
  for (int s = 0; s < splits; ++s) {
    const float ms = part_ml[(base + s) * 2];
    gl += ms == -INFINITY ? 0.f : part_ml[(base + s) * 2 + 1] * exp2f(ms - gm);
  }
  const float inv = gl > 0.f ? 1.f / gl : 0.f;
  for (int c = threadIdx.x; c < width; c += blockDim.x) {
    float v = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float ms = part_ml[(base + s) * 2];
      if (ms != -INFINITY) v += part_o[(base + s) * width + c] * exp2f(ms - gm);
    }
    o[(long long)blockIdx.x * width + c] = __float2bfloat16(v * inv);
  }
}

void launch_latent_merge(const float* part_o, const float* part_ml, __nv_bfloat16* o, int items, int splits, int width,
                         cudaStream_t st) {
  launch_dep(latent_merge_kernel, items, 128, 0, st, part_o, part_ml, o, splits, width);
}

template <int KT, int NT, int HG>
static int launch_latent_decode(const LatentDecodeParams& p, cudaStream_t st) {
  constexpr int smem = LatentDecodeSmem<KT>::bytes(HG);
  auto kern = latent_decode_kernel<KT, NT, HG>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
    configured = true;
  }
  launch_dep(kern, dim3(p.rows, (p.heads + HG * 16 - 1) / (HG * 16), p.splits), 256 * HG, smem, st, p);
  if (p.splits > 1)
    launch_latent_merge(p.part_o, p.part_ml, p.o, p.rows * p.heads, p.splits, p.vwidth, st);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <int KT, int NT>
static int launch_latent_decode_heads(const LatentDecodeParams& p, cudaStream_t st) {
  return p.heads > 16 ? launch_latent_decode<KT, NT, 2>(p, st) : launch_latent_decode<KT, NT, 1>(p, st);
}

}  // namespace b200

using namespace b200;

extern "C" int b200_latent_norm_append(const void* proj, long long ld_proj, const void* wq, const void* wkv, void* cq,
                                       long long ld_cq, void* cache, const long long* slots, int rows, int q_rank,
                                       int kv_rank, int width, long long num_slots, float eps, int f32, uint32_t* status,
                                       cudaStream_t st) {
  if (rows <= 0) return 0;
  if (q_rank <= 0 || kv_rank <= 0 || width < kv_rank) return -10;
  const bool vec = q_rank % 4 == 0 && kv_rank % 4 == 0 && ld_proj % 4 == 0 && ld_cq % 4 == 0 && width % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(cq) | reinterpret_cast<uintptr_t>(cache) |
                     reinterpret_cast<uintptr_t>(wq) | reinterpret_cast<uintptr_t>(wkv)) & 15) == 0;
  // few rows: a warp per block, so that they spread over the SMs
  const int warps = rows >= 148 * 8 ? 8 : 1;
  const unsigned grid = (unsigned)((rows + warps - 1) / warps);
#define LATENT_NORM(T, V)                                                                                               \
  launch_dep(latent_norm_append_kernel<T, V>, grid, warps * 32, 0, st, (const T*)proj, ld_proj, (const T*)wq,           \
             (const T*)wkv, (T*)cq, ld_cq, (T*)cache, slots, rows, q_rank, kv_rank, width, num_slots, eps, status)
  if (f32) {
    if (vec) LATENT_NORM(float, 4);
    else LATENT_NORM(float, 1);
  } else {
    if (vec) LATENT_NORM(__nv_bfloat16, 4);
    else LATENT_NORM(__nv_bfloat16, 1);
  }
#undef LATENT_NORM
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// See LatentRotateParams.  kv_rank <= vwidth <= width - rot; kv_col, k_col negative: the cache keeps what it has.
extern "C" int b200_latent_rotate(void* q, long long ld_q, const void* kv, long long ld_kv, int q_col, int q_pitch, int kv_col, int k_col, const void* wkv, void* ql,
                                  int absorbed, void* cache, const float* cos_sin, const int* positions, const long long* slots,
                                  int rows, int heads, int kv_rank, int vwidth, int width, int rot, int ctx, long long num_slots,
                                  float eps, int f32, uint32_t* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (heads <= 0 || rot <= 0 || (rot & 1) || q_pitch < rot || kv_rank <= 0 || vwidth < kv_rank || width < vwidth + rot ||
      cos_sin == nullptr || ((kv_col >= 0 || k_col >= 0) && kv == nullptr) || (kv_col >= 0 && wkv == nullptr) || (absorbed > 0 && ql == nullptr))
    return -10;
  LatentRotateParams p;
  p.q = q; p.ld_q = ld_q; p.kv = kv; p.ld_kv = ld_kv; p.q_col = q_col; p.q_pitch = q_pitch; p.kv_col = kv_col; p.k_col = k_col; p.wkv = wkv; p.ql = ql;
  p.cache = cache; p.cos_sin = cos_sin; p.positions = positions; p.slots = slots; p.rows = rows; p.absorbed = absorbed;
  p.heads = heads; p.kv_rank = kv_rank; p.vwidth = vwidth; p.width = width; p.rot = rot; p.ctx = ctx; p.num_slots = num_slots;
  p.eps = eps; p.status = status;
  const bool vec = (rot | kv_rank | q_pitch | q_col | vwidth | width) % 4 == 0 && (kv_col < 0 || kv_col % 4 == 0) &&
                   (k_col < 0 || k_col % 4 == 0) && (ld_q | ld_kv) % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(ql) | reinterpret_cast<uintptr_t>(cache) |
                     reinterpret_cast<uintptr_t>(wkv)) & 15) == 0;
  const bool wide = vec && !f32 && (rot | q_pitch | q_col | vwidth | width) % 8 == 0 && (k_col < 0 || k_col % 8 == 0) && (ld_q | ld_kv) % 8 == 0 &&
                    (reinterpret_cast<uintptr_t>(cos_sin) & 15) == 0;
  int threads = 32 + (heads * (rot / (wide ? 8 : (vec ? 4 : 2))) + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  if (wide) {
    launch_dep(latent_rotate_kernel<__nv_bfloat16, 8>, rows, threads, 0, st, p);
  } else if (f32) {
    if (vec) launch_dep(latent_rotate_kernel<float, 4>, rows, threads, 0, st, p);
    else launch_dep(latent_rotate_kernel<float, 2>, rows, threads, 0, st, p);
  } else {
    if (vec) launch_dep(latent_rotate_kernel<__nv_bfloat16, 4>, rows, threads, 0, st, p);
    else launch_dep(latent_rotate_kernel<__nv_bfloat16, 2>, rows, threads, 0, st, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// bf16 caches only (the packed latents feed the tensor-core prefill).
extern "C" int b200_latent_gather(const void* cache, void* out, const int* cu_k, const int* first_k, const int* tables,
                                  int portions, int total_rows, int max_pages, int page_size, int num_pages, int width,
                                  uint32_t* status, cudaStream_t st) {
  if (portions <= 0 || total_rows <= 0) return 0;
  if (width % 8 || (reinterpret_cast<uintptr_t>(cache) & 15) || (reinterpret_cast<uintptr_t>(out) & 15)) return -10;
  const long long n = (long long)total_rows * (width / 8);
  long long blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  launch_dep(latent_gather_kernel<__nv_bfloat16>, (unsigned)blocks, 256, 0, st, (const __nv_bfloat16*)cache,
             (__nv_bfloat16*)out, cu_k, first_k, tables, portions, max_pages, page_size, num_pages, width, width / 8, status);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// window <= 0: no window.  row_seq null: row i uses line i of the tables.
extern "C" int b200_latent_attn_rows(const void* q, const void* cache, void* o, const int* row_seq, const int* positions,
                                     const long long* slots, const int* tables, int seqs, int rows, int heads, int width, int vwidth,
                                     int max_pages, int page_size, int num_pages, int window, float scale, int f32,
                                     uint32_t* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (heads <= 0 || width <= 0 || vwidth <= 0 || vwidth > width || page_size <= 0 || width > 6144) return -10;
  const unsigned grid = (unsigned)(((long long)rows * heads + 3) / 4);
  const size_t smem = 4ull * 2 * width * sizeof(float);
  if (f32) {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(latent_attn_rows_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 (int)smem) != cudaSuccess)
      return -3;
    launch_dep(latent_attn_rows_kernel<float>, grid, 128, smem, st, (const float*)q, (const float*)cache, (float*)o, row_seq,
               positions, slots, tables, seqs, rows, heads, width, vwidth, max_pages, page_size, num_pages, window, scale, status);
  } else {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(latent_attn_rows_kernel<__nv_bfloat16>,
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return -3;
    launch_dep(latent_attn_rows_kernel<__nv_bfloat16>, grid, 128, smem, st, (const __nv_bfloat16*)q,
               (const __nv_bfloat16*)cache, (__nv_bfloat16*)o, row_seq, positions, slots, tables, seqs, rows, heads, width,
               vwidth, max_pages, page_size, num_pages, window, scale, status);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// Decode on the tensor cores: bf16, one query row per line of the tables, width and vwidth multiples of 8, vwidth up to 512, width up to
// 576.  splits > 1 needs part_o (rows * heads * splits * vwidth floats) and part_ml (rows * heads * splits * 2 floats).
extern "C" int b200_latent_decode(const void* q, const void* cache, void* o, float* part_o, float* part_ml,
                                  const int* positions, const long long* slots, const int* tables, int rows, int heads,
                                  int width, int vwidth, int max_pages, int page_size, int num_pages, int window, int splits,
                                  float scale, uint32_t* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (width % 8 || vwidth % 8 || vwidth <= 0 || vwidth > 512 || width < vwidth || width > 576 || heads <= 0 || page_size <= 0 ||
      splits < 1 || splits > 65535)
    return -10;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(o)) & 15) return -10;
  if (splits > 1 && (part_o == nullptr || part_ml == nullptr)) return -11;
  LatentDecodeParams p;
  p.q = (const __nv_bfloat16*)q; p.cache = (const __nv_bfloat16*)cache; p.o = (__nv_bfloat16*)o;
  p.part_o = part_o; p.part_ml = part_ml; p.positions = positions; p.slots = slots; p.tables = tables;
  p.rows = rows; p.heads = heads; p.width = width; p.vwidth = vwidth; p.max_pages = max_pages; p.page_size = page_size;
  p.num_pages = num_pages; p.window = window; p.splits = splits; p.scale_log2 = scale * 1.4426950408889634f;
  p.status = status;
  if (width <= 128) return launch_latent_decode_heads<2, 2>(p, st);
  if (width <= 256) return launch_latent_decode_heads<4, 4>(p, st);
  if (width <= 320 && vwidth <= 256) return launch_latent_decode_heads<5, 4>(p, st);
  if (width <= 512) return launch_latent_decode_heads<8, 8>(p, st);
  return launch_latent_decode_heads<9, 8>(p, st);
}
