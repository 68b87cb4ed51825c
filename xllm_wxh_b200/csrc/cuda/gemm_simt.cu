// C[M,N] = A[M,K] W[N,K]^T on the fp32 pipe, for what the tensor-core GEMMs do not serve: fp32 operands (true 32-bit
// arithmetic, no reduced-precision products), and bf16 shapes whose rows are not 16-byte aligned.  64 x 64 output tiles,
// 256 threads with 4 x 4 outputs each, K in steps of 16 through shared memory.
//
// Grouped (expert) mode reads the same tile table as the tensor-core kernel (gemm_bf16.cu) and can fetch its A rows
// through the expert sort's source index, which saves the separate gather.
#include "vec8.cuh"

namespace xl_simt {
using namespace xl;

constexpr int BM = 64, BN = 64, BK = 16;

struct Tiles {
  const int* tile_expert;
  const int* tile_row0;
  const int* tile_row_end;
  const int* num_m_tiles;      // null: plain GEMM
  const int* row_src;          // null: A row = row; else A row = row_src[row] / row_div
  int row_div;
};
struct Epi {
  const void* bias;            // [N] in the operands' type, or null
  int act;                     // ACT_NONE / ACT_RELU2 / ACT_TANH / ACT_SOFTCAP, applied after the bias
  float cap;                   // ACT_SOFTCAP
  long a_step, w_step, c_step; // batched (blockIdx.z): element offsets from one matrix to the next
};

template <typename T, typename TO>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const T* __restrict__ A, const T* __restrict__ W, TO* __restrict__ C, int M,
                                                        int N, int K, long lda, long ldw, long ldc, const Tiles g, const Epi epi) {
  __shared__ float sA[BK][BM + 4], sW[BK][BN + 4];
  int m0 = blockIdx.x * BM, m_end = M;
  A += blockIdx.z * epi.a_step;
  W += blockIdx.z * epi.w_step;
  C += blockIdx.z * epi.c_step;
  const int n0 = blockIdx.y * BN;
  if (g.num_m_tiles) {                           // 128-row tiles of one expert each, two blocks per tile
    const int tile = blockIdx.x >> 1;
    if (tile >= *g.num_m_tiles) return;
    m0 = g.tile_row0[tile] + (blockIdx.x & 1) * BM;
    m_end = min(g.tile_row_end[tile], g.tile_row0[tile] + 128);
    W += size_t(g.tile_expert[tile]) * N * ldw;
  }
  if (m0 >= m_end) return;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;     // loader: row 0..63, four consecutive k
  const int ar = m0 + lr;
  const T* a_row = nullptr;
  if (ar < m_end) a_row = A + size_t(g.row_src ? g.row_src[ar] / g.row_div : ar) * lda;
  const T* w_row = n0 + lr < N ? W + size_t(n0 + lr) * ldw : nullptr;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      sA[lk + j][lr] = (a_row && k < K) ? to_f32(a_row[k]) : 0.f;
      sW[lk + j][lr] = (w_row && k < K) ? to_f32(w_row[k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sA[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&sW[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= m_end) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      const float b = epi.bias ? to_f32(static_cast<const T*>(epi.bias)[n]) : 0.f;
      from_f32(C + size_t(m) * ldc + n, plain_act(acc[i][j] + b, epi.act, epi.cap));
    }
  }
}

template <typename T, typename TO>
static int launch(const void* A, const void* W, void* C, int M, int N, int K, long lda, long ldw, long ldc, const Tiles& g,
                  const Epi& epi, int m_blocks, cudaStream_t st, int batch = 1) {
  const dim3 grid(m_blocks, (N + BN - 1) / BN, batch);
  if (grid.y > 65535 || batch > 65535) return -2;
  gemm_simt_kernel<T, TO><<<grid, 256, 0, st>>>(static_cast<const T*>(A), static_cast<const T*>(W), static_cast<TO*>(C), M, N, K, lda, ldw,
                                                ldc, g, epi);
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

static int dispatch(const void* A, const void* W, void* C, int M, int N, int K, long lda, long ldw, long ldc, int in_f32, int out_f32,
                    const Tiles& g, const Epi& epi, int m_blocks, cudaStream_t st, int batch = 1) {
  if (in_f32) return out_f32 ? launch<float, float>(A, W, C, M, N, K, lda, ldw, ldc, g, epi, m_blocks, st, batch) : -2;
  if (out_f32) return launch<__nv_bfloat16, float>(A, W, C, M, N, K, lda, ldw, ldc, g, epi, m_blocks, st, batch);
  return launch<__nv_bfloat16, __nv_bfloat16>(A, W, C, M, N, K, lda, ldw, ldc, g, epi, m_blocks, st, batch);
}

}  // namespace xl_simt

// in_f32: A and W are fp32 (else bf16); out_f32: C is fp32 (else bf16).  C = act(A W^T + bias), bias [N] or null.
XL_API int xl_gemm_simt(const void* A, const void* W, void* C, const void* bias, int act, float cap, int M, int N, int K, long lda, long ldw,
                        long ldc, int in_f32, int out_f32, void* stream) {
  if (M <= 0 || N <= 0) return 0;
  xl_simt::Tiles g = {};
  const xl_simt::Epi epi{bias, act, cap, 0, 0, 0};
  return xl_simt::dispatch(A, W, C, M, N, K, lda, ldw, ldc, in_f32, out_f32, g, epi, (M + xl_simt::BM - 1) / xl_simt::BM,
                           static_cast<cudaStream_t>(stream));
}

// `batch` products of the same shape, whose A, W and C lie a_step, w_step and c_step elements apart.
XL_API int xl_gemm_simt_batched(const void* A, const void* W, void* C, int batch, int M, int N, int K, long lda, long ldw, long ldc,
                                long a_step, long w_step, long c_step, int f32, void* stream) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  xl_simt::Tiles g = {};
  const xl_simt::Epi epi{nullptr, xl::ACT_NONE, 0.f, a_step, w_step, c_step};
  return xl_simt::dispatch(A, W, C, M, N, K, lda, ldw, ldc, f32, f32, g, epi, (M + xl_simt::BM - 1) / xl_simt::BM,
                           static_cast<cudaStream_t>(stream), batch);
}

// Grouped form: W [E, N, K] dense, the tile table of `xl_moe_sort`; `row_src` (may be null) maps a sorted row to
// row_src[row] / row_div of A.  `act` as in xl_gemm_simt.
XL_API int xl_grouped_gemm_simt(const void* A, const void* W, void* C, int N, int K, long lda, long ldc, const void* tile_expert,
                                const void* tile_row0, const void* tile_row_end, const void* num_m_tiles, int max_m_tiles,
                                const void* row_src, int row_div, int act, int f32, void* stream) {
  if (max_m_tiles <= 0 || N <= 0) return 0;
  xl_simt::Tiles g;
  g.tile_expert = static_cast<const int*>(tile_expert);
  g.tile_row0 = static_cast<const int*>(tile_row0);
  g.tile_row_end = static_cast<const int*>(tile_row_end);
  g.num_m_tiles = static_cast<const int*>(num_m_tiles);
  g.row_src = static_cast<const int*>(row_src);
  g.row_div = row_div < 1 ? 1 : row_div;
  return xl_simt::dispatch(A, W, C, 0, N, K, lda, K, ldc, f32, f32, g, xl_simt::Epi{nullptr, act, 0.f, 0, 0, 0}, 2 * max_m_tiles,
                           static_cast<cudaStream_t>(stream));
}
