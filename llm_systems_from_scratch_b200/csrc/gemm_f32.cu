// fp32 GEMM on the FMA pipes, D[m, n] = sum_k A[m, k] B[n, k], for models that run in 32-bit: the tensor cores have no
// full fp32 mode.  Same three problem kinds as the bf16 kernel (one problem, one group of B rows per 128-row tile of A,
// or one problem per head side by side); no alignment requirements.
#include "gemm_common.cuh"

namespace b200 {

constexpr int SG_TILE = 64, SG_K = 16;

struct GemmF32Params {
  const float *A, *B;
  float* C;
  int M, N, K;
  long long lda, ldb, ldc;
  int accumulate;
  const int* tile_group;       // per 128 rows of A
  int group_rows, a_step, c_step;
  int finished;
  GemmFinish finish;
};

__global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32Params p) {
  pdl_sync();
  __shared__ float sa[SG_K][SG_TILE + 4], sb[SG_K][SG_TILE + 4];
  const int m0 = blockIdx.y * SG_TILE, n0 = blockIdx.x * SG_TILE;
  int group = blockIdx.z;
  if (p.tile_group != nullptr) {
    group = p.tile_group[m0 / 128];
    if (group < 0) return;
  }
  const float* A = p.A + (long long)blockIdx.z * p.a_step;
  const float* B = p.B + (long long)group * p.group_rows * p.ldb;
  float* C = p.C + (long long)blockIdx.z * p.c_step;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += SG_K) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (threadIdx.x >> 4) + i * 16, k = threadIdx.x & 15;
      sa[k][r] = (m0 + r < p.M && k0 + k < p.K) ? A[(long long)(m0 + r) * p.lda + k0 + k] : 0.f;
      sb[k][r] = (n0 + r < p.N && k0 + k < p.K) ? B[(long long)(n0 + r) * p.ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SG_K; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sa[k][ty * 4 + i]; b[i] = sb[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < p.M && n < p.N) {
        float* c = C + (long long)m * p.ldc + n;
        float v = acc[i][j];
        if (p.finished) v = finish_act(p.finish.alpha * (v + (p.finish.bias != nullptr ? p.finish.bias[n] : 0.f)), p.finish.act, p.finish.cap);
        *c = p.accumulate ? *c + v : v;
      }
    }
}

}  // namespace b200

using namespace b200;

// accumulate: C += A B^T.  tile_group / batch as in b200_gemm_bf16_grouped (batch <= 1 and no tile_group: one problem).
// finish: null, or what to do with the sums first (a bias is that of a single problem).
extern "C" int b200_gemm_f32(const float* A, const float* B, float* C, int M, int N, int K, long long lda, long long ldb,
                             long long ldc, int accumulate, const int* tile_group, int group_rows, int batch, int a_step,
                             int c_step, const GemmFinish* finish, cudaStream_t st) {
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  if (tile_group != nullptr && (batch > 1 || M % 128)) return -12;
  GemmF32Params p;
  p.A = A; p.B = B; p.C = C; p.M = M; p.N = N; p.K = K; p.lda = lda; p.ldb = ldb; p.ldc = ldc;
  p.accumulate = accumulate; p.tile_group = tile_group;
  p.group_rows = group_rows; p.a_step = a_step; p.c_step = c_step; p.finished = finish != nullptr;
  if (finish != nullptr) p.finish = *finish;
  const dim3 grid((N + SG_TILE - 1) / SG_TILE, (M + SG_TILE - 1) / SG_TILE, batch > 1 ? batch : 1);
  if (grid.y > 65535 || grid.z > 65535) return -13;
  launch_dep(gemm_f32_kernel, grid, 256, 0, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
