// Latent-attention decode on tcgen05: one query row per request against its window of paged latents (see
// latent_attention.cu for the mechanism and for the general and mma.sync kernels).
//
// With H heads a cached latent takes 4 H FLOP per element; mma.sync runs out of tensor throughput before the memory system
// does.  Here the TOKENS are the M dimension, so the heads only have to fill N (16, 32 or 64):
//     S^T (128 tokens x heads)        = C (tokens x latent)  Q^T            A = C, K-major
//     O^T (128 latent dims x heads)  += C^T (latent x tokens) P^T           A = C, MN-major, the same shared memory
// A rotated key part behind the latent (up to 64 columns) is a stage of its own that only takes part in the scores.  It comes first in
// a tile, so that its place in the ring is free again before the tile's last latents need one.
// One CTA = one request and one split of its window, in tiles of 128 tokens that start on page borders.
//   warp 0      TMA producer: pages -> a ring of stages of 128 tokens x 128 latent columns (one box per page and 64 columns;
//               the lanes issue one page each; pages of 64 tokens keep the number of boxes small)
//   warp 1      MMA issuer: S^T as the stages of a tile land; then O^T stage by stage, which frees them
//   warps 2-9   softmax: a thread holds one token's scores of half of the heads; maxima go across lanes and warps, P^T (heads
//               x tokens, bf16) goes to shared memory; O^T is rescaled in tensor memory only when a maximum moved by more than
//               2^8.  They also zero the rows of the last tile that lie past the request's last token.
#include "typed.cuh"

namespace b200 {

int make_tmap_bf16_2d(CUtensorMap* tm, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_cols,
                      uint32_t box_rows);

struct LatentTcParams {
  const __nv_bfloat16* q;       // (rows, heads * width)
  __nv_bfloat16* o;             // (rows, heads * vwidth)
  float* part_o;                // (rows, heads, splits, vwidth) when splits > 1
  float* part_ml;               // (rows, heads, splits, 2)
  const int* positions;
  const long long* slots;
  const int* tables;
  int rows, heads, width, vwidth, max_pages, page_size, num_pages, window, splits;
  float scale_log2;
  uint32_t* status;
};

constexpr int LT_TILE = 128;
constexpr int LT_SOFTMAX = 256;                       // threads: four warps per half of the heads
constexpr int LT_THREADS = 64 + LT_SOFTMAX;

__device__ __forceinline__ float lt_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int HN>
struct LatentTcSmem {
  static constexpr int STAGES = HN == 16 ? 6 : (HN == 32 ? 5 : 4);
  static constexpr int STAGE = 32768;                    // two panels of 128 tokens x 64 latent columns
  static constexpr int OFF_Q = STAGES * STAGE;           // panels of HN rows x 128 bytes, up to 9
  static constexpr int OFF_P = OFF_Q + 9 * HN * 128;     // two panels of HN rows x 64 tokens
  static constexpr int OFF_MAX = OFF_P + 2 * HN * 128;   // [4][HN] floats
  static constexpr int OFF_RUN = OFF_MAX + 4 * HN * 4;   // m [HN], alpha [HN], need
  static constexpr int OFF_BAR = OFF_RUN + 2 * HN * 4 + 16;
  static constexpr int TOTAL = OFF_BAR + (2 * STAGES + 3) * 8 + 16 + 1024;
  static constexpr int TMEM_COLS = HN == 16 ? 128 : (HN == 32 ? 256 : 512);   // S: HN, O: up to 4 HN
};

// Maximum over the warp's lanes of N values per lane, N a power of two <= 32: afterwards lane l holds that of value l % N
// (for N < 32 in several lanes).  Halving exchange: N - 1 + log2(32 / N) shuffles instead of 5 N.
template <int N>
__device__ __forceinline__ float warp_max_of(float (&v)[N]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int w = N / 2; w > 0; w >>= 1) {
    const bool up = (lane & w) != 0;
#pragma unroll
    for (int i = 0; i < w; ++i) {
      const float keep = up ? v[i + w] : v[i], give = up ? v[i] : v[i + w];
      v[i] = fmaxf(keep, __shfl_xor_sync(0xffffffffu, give, w));
    }
  }
  float m = v[0];
#pragma unroll
  for (int o = N; o < 32; o <<= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
  return m;
}
template <int N>
__device__ __forceinline__ float warp_sum_of(float (&v)[N]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int w = N / 2; w > 0; w >>= 1) {
    const bool up = (lane & w) != 0;
#pragma unroll
    for (int i = 0; i < w; ++i) {
      const float keep = up ? v[i + w] : v[i], give = up ? v[i] : v[i + w];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, w);
    }
  }
  float m = v[0];
#pragma unroll
  for (int o = N; o < 32; o <<= 1) m += __shfl_xor_sync(0xffffffffu, m, o);
  return m;
}

__device__ __forceinline__ void tmem_ld_32x8(uint32_t taddr, uint32_t (&r)[8]) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0, %1, %2, %3, %4, %5, %6, %7}, [%8];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
               : "r"(taddr)
               : "memory");
}
__device__ __forceinline__ void tmem_st_32x8(uint32_t taddr, const uint32_t (&r)[8]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"r"(taddr), "r"(r[0]),
               "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7])
               : "memory");
}
__device__ __forceinline__ void softmax_barrier() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

template <int HN>
__global__ void __launch_bounds__(LT_THREADS, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tm_cache, const LatentTcParams p) {
  using L = LatentTcSmem<HN>;
  constexpr int ST = L::STAGES, HH = HN / 2;      // ring stages, heads of a softmax thread
  extern __shared__ uint8_t lt_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lt_raw) + 1023) & ~uintptr_t(1023));
  float* smax = reinterpret_cast<float*>(smem + L::OFF_MAX);
  float* srun = reinterpret_cast<float*>(smem + L::OFF_RUN);
  float* salpha = srun + HN;
  volatile int* sneed = reinterpret_cast<volatile int*>(salpha + HN);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::OFF_BAR);
  uint64_t *full = bars, *empty = bars + ST, *s_full = bars + 2 * ST, *p_full = s_full + 1, *o_full = s_full + 2;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(bars + 2 * ST + 3);
  volatile uint32_t* abort_word = tmem_holder + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    for (int i = 0; i < ST; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(s_full, 1);
    mbar_init(p_full, LT_SOFTMAX);
    mbar_init(o_full, 1);
    *abort_word = 0;
    fence_barrier_init();
    prefetch_tensormap(&tm_cache);
  }
  if (warp == 1) {
    tmem_alloc(tmem_holder, L::TMEM_COLS);
    tmem_relinquish();
  }
  pdl_sync();
  const int row = blockIdx.x, split = blockIdx.y;
  const int pos = p.positions[row];
  const bool live = p.slots[row] >= 0 && pos >= 0;
  const int lo = (p.window > 0 && pos - p.window + 1 > 0) ? pos - p.window + 1 : 0;
  const int base = lo / p.page_size * p.page_size;              // tiles start on page borders
  const int total = live ? (pos + 1 - base + LT_TILE - 1) / LT_TILE : 0;
  const int per = (total + p.splits - 1) / p.splits;
  const int i0 = min(total, split * per), tiles = min(total, i0 + per) - i0;
  const int nv = p.vwidth / 128, nr = p.width > p.vwidth ? 1 : 0, nb = nv + nr;      // stages per tile: rotated part, latents
  const int t_first = base + i0 * LT_TILE;

  if (warp >= 2) {                                              // queries: HN rows, zero beyond the heads
    const int vecs = (p.width + 63) / 64 * 8;                   // whole panels, zero beyond the width
    for (int i = threadIdx.x - 64; i < HN * vecs; i += LT_SOFTMAX) {
      const int h = i / vecs, v = i - h * vecs;
      uint4 x = make_uint4(0, 0, 0, 0);
      if (h < p.heads && v * 8 < p.width) x = *reinterpret_cast<const uint4*>(p.q + ((long long)row * p.heads + h) * p.width + v * 8);
      *reinterpret_cast<uint4*>(smem + L::OFF_Q + (v >> 3) * (HN * 128) + h * 128 + (((v & 7) ^ (h & 7)) << 4)) = x;
    }
    if (threadIdx.x - 64 < HN) srun[threadIdx.x - 64] = -INFINITY;
    fence_proxy_async_smem();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_holder;                           // S^T: columns [0, HN); O^T of stage b: [HN (1 + b), ...)

  if (warp == 0) {
    // ------------------------------------------------------------------------------------------ TMA producer
    const int pages = LT_TILE / p.page_size;                    // per tile, <= 16
    const int last_page = live ? pos / p.page_size : 0;
    bool ok = true;
    for (int i = 0; i < tiles && ok; ++i) {
      int page = 0;
      if (lane < pages) {
        const int pg = min((t_first + i * LT_TILE) / p.page_size + lane, last_page);    // past the end: something valid
        page = pg < p.max_pages ? p.tables[(long long)row * p.max_pages + pg] : -1;
        if ((unsigned)page >= (unsigned)p.num_pages) {
          report_bad_arg(p.status, 12);
          page = 0;
        }
      }
      for (int b = 0; b < nb; ++b) {
        const int g = i * nb + b, st = g % ST;
        if (!mbar_wait(&empty[st], ((g / ST) & 1) ^ 1, abort_word)) {
          *abort_word = ERR_WAIT_EMPTY;
          ok = false;
          break;
        }
        const bool rot = b < nr;
        if (lane == 0) mbar_expect_tx(&full[st], rot ? L::STAGE / 2 : L::STAGE);
        __syncwarp();
        if (lane < pages) {
          uint8_t* dst = smem + st * L::STAGE + lane * p.page_size * 128;
          const int col = rot ? p.vwidth : (b - nr) * 128;
          tma_load_2d(dst, &tm_cache, &full[st], col, page * p.page_size);
          if (!rot) tma_load_2d(dst + 16384, &tm_cache, &full[st], col + 64, page * p.page_size);
        }
        __syncwarp();
      }
    }
  } else if (warp == 1) {
    // -------------------------------------------------------------------------------------------- MMA issuer
    if (elect_one()) {
      constexpr uint32_t id_s = make_idesc_bf16(128, HN, false, false), id_o = make_idesc_bf16(128, HN, true, false);
      bool ok = true;
      for (int i = 0; i < tiles && ok; ++i) {
        for (int b = 0; b < nb && ok; ++b) {
          const int g = i * nb + b, st = g % ST;
          ok = mbar_wait(&full[st], (g / ST) & 1, abort_word);
          if (!ok) break;
          tc_fence_after();
          const uint64_t c = make_smem_desc(smem_u32(smem + st * L::STAGE), 16, 1024);
          const bool rot = b < nr;
          const uint64_t q = make_smem_desc(smem_u32(smem + L::OFF_Q + (rot ? nv : b - nr) * 2 * HN * 128), 16, 1024);
          const int ksteps = rot ? (p.width - p.vwidth + 15) / 16 : 8;
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            if (k >= ksteps) break;
            umma_f16_ss(tmem, c + (uint32_t)(((k / 4) * 16384 + (k % 4) * 32) >> 4),
                        q + (uint32_t)(((k / 4) * HN * 128 + (k % 4) * 32) >> 4), id_s, (b | k) ? 1u : 0u);
          }
          if (rot) umma_commit(&empty[st]);
        }
        if (!ok) break;
        umma_commit(s_full);
        ok = mbar_wait(p_full, i & 1, abort_word);
        if (!ok) break;
        tc_fence_after();
        const uint64_t pt = make_smem_desc(smem_u32(smem + L::OFF_P), 16, 1024);
        for (int b = 0; b < nv; ++b) {
          const int st = (i * nb + nr + b) % ST;
          const uint64_t ct = make_smem_desc(smem_u32(smem + st * L::STAGE), 16384, 1024);
#pragma unroll
          for (int k = 0; k < 8; ++k)
            umma_f16_ss(tmem + HN * (1 + b), ct + (uint32_t)(k * 128),
                        pt + (uint32_t)(((k / 4) * HN * 128 + (k % 4) * 32) >> 4), id_o, (i | k) ? 1u : 0u);
          umma_commit(&empty[st]);
        }
      }
      if (ok && tiles > 0) umma_commit(o_full);
      if (!ok) *abort_word = ERR_WAIT_FULL;
    }
  } else {
    // ----------------------------------------------------------------------------------------------- softmax
    const int quarter = warp & 3, r = quarter * 32 + lane;      // token of the tile; latent dim of a stage in the end
    const int half = (warp - 2) >> 2, hb = half * HH;           // this thread's heads: [hb, hb + HH)
    const int tid = threadIdx.x - 64;
    const uint32_t lane_addr = uint32_t(quarter * 32) << 16;
    bool ok = true;
    float l[HH];
#pragma unroll
    for (int h = 0; h < HH; ++h) l[h] = 0.f;
    uint8_t* p_base = smem + L::OFF_P + (r >> 6) * (HN * 128) + hb * 128 + (r & 7) * 2;    // P^T: row = head, column = token
    const int p_piece = (r >> 3) & 7;
    // HH columns of tensor memory, eight at a time
    auto load_cols = [&](uint32_t col, float (&v)[HH]) __attribute__((always_inline)) {
#pragma unroll
      for (int c = 0; c < HH / 8; ++c) {
        uint32_t raw[8];
        tmem_ld_32x8(tmem + lane_addr + col + c * 8, raw);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 8; ++j) v[c * 8 + j] = __uint_as_float(raw[j]);
      }
    };
    for (int i = 0; i < tiles; ++i) {
      const int t = t_first + i * LT_TILE + r;
      const bool seen = t >= lo && t <= pos;
      if (!mbar_wait(s_full, i & 1, abort_word)) { ok = false; *abort_word = ERR_WAIT_MISC; }
      tc_fence_after();
      if (t > pos) {                   // never written by this request: zero, so that it cannot reach O even as 0 * NaN
        for (int b = 0; b < nv; ++b) {
          uint8_t* c = smem + ((i * nb + nr + b) % ST) * L::STAGE + half * 16384 + r * 128;
#pragma unroll
          for (int v = 0; v < 8; ++v) *reinterpret_cast<uint4*>(c + v * 16) = make_uint4(0, 0, 0, 0);
        }
      }
      __syncwarp();
      float s[HH];
      load_cols(hb, s);
      float v[HH];
#pragma unroll
      for (int j = 0; j < HH; ++j) {
        s[j] = seen ? s[j] * p.scale_log2 : -INFINITY;
        v[j] = s[j];
      }
      {
        const float m = warp_max_of<HH>(v);
        if (lane < HH) smax[quarter * HN + hb + lane] = m;
      }
      if (tid == 0) *sneed = 0;
      softmax_barrier();
      if (tid < HN) {
        const float mx = fmaxf(fmaxf(smax[tid], smax[HN + tid]), fmaxf(smax[2 * HN + tid], smax[3 * HN + tid]));
        const float old = srun[tid];
        const float now = mx > old + 8.f ? mx : old;            // finite: every tile holds a token that is seen
        srun[tid] = now;
        salpha[tid] = lt_exp2(old - now);
        if (now != old) *sneed = 1;
      }
      softmax_barrier();
      const bool need = *sneed != 0;
      float alpha[HH];
#pragma unroll
      for (int h = 0; h < HH; h += 4) {
        const float4 a4 = *reinterpret_cast<const float4*>(salpha + hb + h), m4 = *reinterpret_cast<const float4*>(srun + hb + h);
        alpha[h] = a4.x; alpha[h + 1] = a4.y; alpha[h + 2] = a4.z; alpha[h + 3] = a4.w;
        s[h] -= m4.x; s[h + 1] -= m4.y; s[h + 2] -= m4.z; s[h + 3] -= m4.w;
      }
#pragma unroll
      for (int h = 0; h < HH; ++h) {
        const float e = lt_exp2(s[h]);
        l[h] = fmaf(l[h], alpha[h], e);
        *reinterpret_cast<__nv_bfloat16*>(p_base + h * 128 + ((p_piece ^ (h & 7)) << 4)) = __float2bfloat16(e);
      }
      if (need && i > 0) {             // S^T(i) was issued after the products of tile i - 1, so those are complete
        for (int b = 0; b < nv; ++b)
#pragma unroll
          for (int c = 0; c < HH / 8; ++c) {
            uint32_t raw[8];
            tmem_ld_32x8(tmem + lane_addr + HN * (1 + b) + hb + c * 8, raw);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 8; ++j) raw[j] = __float_as_uint(__uint_as_float(raw[j]) * alpha[c * 8 + j]);
            tmem_st_32x8(tmem + lane_addr + HN * (1 + b) + hb + c * 8, raw);
          }
        tmem_st_wait();
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(p_full);
    }
    // sums over the tokens: across lanes, then warps
    softmax_barrier();
    {
      const float sum = warp_sum_of<HH>(l);
      if (lane < HH) smax[quarter * HN + hb + lane] = sum;
    }
    softmax_barrier();
    if (tid < HN) {
      const float sum = (smax[tid] + smax[HN + tid]) + (smax[2 * HN + tid] + smax[3 * HN + tid]);
      salpha[tid] = sum > 0.f ? 1.f / sum : 0.f;
      if (p.splits > 1 && tid < p.heads) {
        float* ml = p.part_ml + (((long long)row * p.heads + tid) * p.splits + split) * 2;
        ml[0] = srun[tid];
        ml[1] = sum;
      }
    }
    softmax_barrier();
    if (tiles > 0 && !mbar_wait(o_full, 0, abort_word)) { ok = false; *abort_word = ERR_WAIT_TMEM_FULL; }
    tc_fence_after();
    for (int b = 0; b < nv; ++b) {
      float x[HH];
      if (tiles > 0 && ok) {
        load_cols(HN * (1 + b) + hb, x);
      } else {
#pragma unroll
        for (int j = 0; j < HH; ++j) x[j] = 0.f;
      }
#pragma unroll
      for (int j = 0; j < HH; ++j) {
        const int h = hb + j;
        if (h >= p.heads) break;
        if (p.splits > 1)
          p.part_o[(((long long)row * p.heads + h) * p.splits + split) * p.vwidth + b * 128 + r] = x[j];
        else
          p.o[((long long)row * p.heads + h) * p.vwidth + b * 128 + r] = __float2bfloat16(x[j] * salpha[h]);
      }
    }
  }
  __syncwarp();
  tc_fence_before();
  __syncthreads();
  if (*abort_word != 0) {
    if (threadIdx.x == 0 && p.status != nullptr) atomicCAS(p.status, 0u, (*abort_word) | (blockIdx.x << 8));
    const uint64_t w0 = globaltimer_ns();
    while (globaltimer_ns() - w0 < 200000ull) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, L::TMEM_COLS);
  }
}

void launch_latent_merge(const float* part_o, const float* part_ml, __nv_bfloat16* o, int items, int splits, int width,
                         cudaStream_t st);

template <int HN>
static int launch_latent_tc(const CUtensorMap& tm, const LatentTcParams& p, cudaStream_t st) {
  auto kern = latent_decode_tc_kernel<HN>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, LatentTcSmem<HN>::TOTAL) != cudaSuccess)
      return -3;
    configured = true;
  }
  launch_dep(kern, dim3(p.rows, p.splits), LT_THREADS, LatentTcSmem<HN>::TOTAL, st, tm, p);
  if (p.splits > 1) launch_latent_merge(p.part_o, p.part_ml, p.o, p.rows * p.heads, p.splits, p.vwidth, st);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace b200

using namespace b200;

// As b200_latent_decode, for vwidths that are multiples of 128 up to 512, widths up to 64 above, at most 64 heads and page sizes
// 8 .. 128 that divide 128.
extern "C" int b200_latent_decode_tc(const void* q, const void* cache, void* o, float* part_o, float* part_ml,
                                     const int* positions, const long long* slots, const int* tables, int rows, int heads,
                                     int width, int vwidth, int max_pages, int page_size, int num_pages, int window, int splits,
                                     float scale, uint32_t* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (vwidth % 128 || vwidth <= 0 || vwidth > 512 || width % 8 || width < vwidth || width > vwidth + 64 || heads <= 0 || heads > 64 || page_size < 8 || page_size > 128 ||
      128 % page_size || splits < 1 || splits > 65535)
    return -10;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(o)) & 15) return -10;
  if (splits > 1 && (part_o == nullptr || part_ml == nullptr)) return -11;
  CUtensorMap tm;
  if (make_tmap_bf16_2d(&tm, cache, (uint64_t)num_pages * page_size, (uint64_t)width, (uint64_t)width, 64, (uint32_t)page_size))
    return -20;
  LatentTcParams p;
  p.q = (const __nv_bfloat16*)q; p.o = (__nv_bfloat16*)o; p.part_o = part_o; p.part_ml = part_ml;
  p.positions = positions; p.slots = slots; p.tables = tables; p.rows = rows; p.heads = heads; p.width = width; p.vwidth = vwidth;
  p.max_pages = max_pages; p.page_size = page_size; p.num_pages = num_pages; p.window = window; p.splits = splits;
  p.scale_log2 = scale * 1.4426950408889634f; p.status = status;
  if (heads <= 16) return launch_latent_tc<16>(tm, p, st);
  if (heads <= 32) return launch_latent_tc<32>(tm, p, st);
  return launch_latent_tc<64>(tm, p, st);
}
