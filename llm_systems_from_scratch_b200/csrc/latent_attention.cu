// Latent attention over a paged cache of latents.  Keys and values of all heads are linear images of one cached vector c
// per token (k_h = W_uk,h c, v_h = W_uv,h c), so a query is moved into latent space first (q'_h = W_uk,h^T q_h, a small
// GEMM per head): score = q'_h . c * scale, and sum_j p_j c_j goes through W_uv,h afterwards.  Every cached byte is then
// read once for all heads.  The mask is a sliding window: position i sees the `window` positions up to and including i.
//
// Cache layout per layer run: (num_pages, page_size, width), width = latent size rounded up to 8 elements, zero padded.
#include "typed.cuh"

namespace b200 {

// Row-wise norms of the two latents of a layer and the append to the cache:
//   cq[row] = rms_norm(proj[row, 0 : q_rank]) * wq,   cache[slot[row]] = rms_norm(proj[row, q_rank : q_rank + kv_rank]) * wkv
template <typename T>
__global__ void __launch_bounds__(256) latent_norm_append_kernel(
    const T* __restrict__ proj, long long ld_proj, const T* __restrict__ wq, const T* __restrict__ wkv, T* __restrict__ cq,
    long long ld_cq, T* __restrict__ cache, const long long* __restrict__ slots, int q_rank, int kv_rank, int width,
    long long num_slots, float eps, uint32_t* __restrict__ status) {
  pdl_sync();
  __shared__ float red[32];
  const int row = blockIdx.x;
  const T* pr = proj + (long long)row * ld_proj;
  const long long slot = slots[row];
  float sq = 0.f, skv = 0.f;
  for (int c = threadIdx.x; c < q_rank; c += blockDim.x) { const float v = to_f(pr[c]); sq += v * v; }
  for (int c = threadIdx.x; c < kv_rank; c += blockDim.x) { const float v = to_f(pr[q_rank + c]); skv += v * v; }
  const float rq = rsqrtf(block_total(sq, red) / (float)q_rank + eps);
  const float rkv = rsqrtf(block_total(skv, red) / (float)kv_rank + eps);
  T* q = cq + (long long)row * ld_cq;
  for (int c = threadIdx.x; c < q_rank; c += blockDim.x) from_f(q[c], to_f(pr[c]) * rq * to_f(wq[c]));
  if (slot < 0) return;                       // padding row of the batch
  if (slot >= num_slots) {
    if (threadIdx.x == 0) report_bad_arg(status, 4);
    return;
  }
  T* dst = cache + slot * width;
  for (int c = threadIdx.x; c < kv_rank; c += blockDim.x) from_f(dst[c], to_f(pr[q_rank + c]) * rkv * to_f(wkv[c]));
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
// q / o: (rows, heads * width).  row_seq[row] names the row's line of `tables`.
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_rows_kernel(
    const T* __restrict__ q, const T* __restrict__ cache, T* __restrict__ o, const int* __restrict__ row_seq,
    const int* __restrict__ positions, const long long* __restrict__ slots, const int* __restrict__ tables, int seqs,
    int rows, int heads, int width, int max_pages, int page_size, int num_pages, int window, float scale,
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
  T* orow = o + ((long long)row * heads + h) * width;
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
      for (int i = lane; i < width; i += 32) acc[i] = acc[i] * a + e * to_f(c[i]);
      m = mn;
    }
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int c = lane; c < width; c += 32) from_f(orow[c], acc[c] * inv);
}

}  // namespace b200

using namespace b200;

extern "C" int b200_latent_norm_append(const void* proj, long long ld_proj, const void* wq, const void* wkv, void* cq,
                                       long long ld_cq, void* cache, const long long* slots, int rows, int q_rank,
                                       int kv_rank, int width, long long num_slots, float eps, int f32, uint32_t* status,
                                       cudaStream_t st) {
  if (rows <= 0) return 0;
  if (q_rank <= 0 || kv_rank <= 0 || width < kv_rank) return -10;
  const int big = q_rank > kv_rank ? q_rank : kv_rank;
  int threads = (big / 4 + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 256 ? 256 : threads);
  if (f32)
    launch_dep(latent_norm_append_kernel<float>, rows, threads, 0, st, (const float*)proj, ld_proj, (const float*)wq,
               (const float*)wkv, (float*)cq, ld_cq, (float*)cache, slots, q_rank, kv_rank, width, num_slots, eps, status);
  else
    launch_dep(latent_norm_append_kernel<__nv_bfloat16>, rows, threads, 0, st, (const __nv_bfloat16*)proj, ld_proj,
               (const __nv_bfloat16*)wq, (const __nv_bfloat16*)wkv, (__nv_bfloat16*)cq, ld_cq, (__nv_bfloat16*)cache,
               slots, q_rank, kv_rank, width, num_slots, eps, status);
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
                                     const long long* slots, const int* tables, int seqs, int rows, int heads, int width,
                                     int max_pages, int page_size, int num_pages, int window, float scale, int f32,
                                     uint32_t* status, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (heads <= 0 || width <= 0 || page_size <= 0 || width > 6144) return -10;
  const unsigned grid = (unsigned)(((long long)rows * heads + 3) / 4);
  const size_t smem = 4ull * 2 * width * sizeof(float);
  if (f32) {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(latent_attn_rows_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 (int)smem) != cudaSuccess)
      return -3;
    launch_dep(latent_attn_rows_kernel<float>, grid, 128, smem, st, (const float*)q, (const float*)cache, (float*)o, row_seq,
               positions, slots, tables, seqs, rows, heads, width, max_pages, page_size, num_pages, window, scale, status);
  } else {
    if (smem > 48 * 1024 && cudaFuncSetAttribute(latent_attn_rows_kernel<__nv_bfloat16>,
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return -3;
    launch_dep(latent_attn_rows_kernel<__nv_bfloat16>, grid, 128, smem, st, (const __nv_bfloat16*)q,
               (const __nv_bfloat16*)cache, (__nv_bfloat16*)o, row_seq, positions, slots, tables, seqs, rows, heads, width,
               max_pages, page_size, num_pages, window, scale, status);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
