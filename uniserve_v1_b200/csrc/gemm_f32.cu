// FP32 linear  out[r, m] = act(sum_k X[r, k] W[g, m, k] + bias[m])  for models served in true
// 32-bit (no reduced-precision tensor mode): FP32 operands, FP32 fused multiply-adds.  Dense,
// or grouped over the expert tile list of moe_route.cu.  A CTA computes 64 rows x 64 features
// from 16-wide K tiles in shared memory, 4 x 4 outputs per thread.
#include "include/us_common.cuh"

namespace {

constexpr int kT = 64, kK = 16;

struct F32Args {
  const float *W, *X, *bias;
  float* out;
  long long ldw, ldx, ldo;
  int w_rows, M, K, rows, act;
  const int *tile_group, *tile_row0, *tile_rows, *num_tiles;
  float act_a, act_b;
};

__device__ __forceinline__ float act_f(float x, int act, float a, float b) {
  if (act == 5) {
    x = fmaxf(x, 0.f);
    return x * x;
  }
  if (act == 6) return fmaf(x > 0.f ? a * x : b, x > 0.f ? x : expm1f(x) - x, 0.5f * x);
  return act == 3 ? 0.5f * x * (1.f + erff(x * 0.70710678118654752f)) : x;
}

__global__ void __launch_bounds__(256) gemm_f32_kernel(const F32Args a) {
  US_PDL_PROLOGUE();
  __shared__ float xs[kK][kT + 4], ws[kK][kT + 4];
  int row_lo, row_hi, group = 0;
  if (a.num_tiles) {
    if ((int)blockIdx.y >= *a.num_tiles) return;
    group = a.tile_group[blockIdx.y];
    row_lo = a.tile_row0[blockIdx.y];
    row_hi = row_lo + a.tile_rows[blockIdx.y];
  } else {
    row_lo = blockIdx.y * kT;
    row_hi = min(a.rows, row_lo + kT);
  }
  const float* W = a.W + (long long)group * a.w_rows * a.ldw;
  const int m0 = blockIdx.x * kT;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  for (int r0 = row_lo; r0 < row_hi; r0 += kT) {
    float acc[4][4] = {};
    for (int k0 = 0; k0 < a.K; k0 += kK) {
      for (int e = threadIdx.x; e < kT * kK; e += 256) {
        const int i = e / kK, k = e - i * kK;
        const bool kin = k0 + k < a.K;
        xs[k][i] = (kin && r0 + i < row_hi) ? a.X[(long long)(r0 + i) * a.ldx + k0 + k] : 0.f;
        ws[k][i] = (kin && m0 + i < a.M) ? W[(long long)(m0 + i) * a.ldw + k0 + k] : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int k = 0; k < kK; ++k) {
        float xv[4], wv[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          xv[i] = xs[k][ty * 4 + i];
          wv[i] = ws[k][tx * 4 + i];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
      }
      __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = r0 + ty * 4 + i;
      if (r >= row_hi) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int m = m0 + tx * 4 + j;
        if (m >= a.M) continue;
        a.out[(long long)r * a.ldo + m] = act_f(acc[i][j] + (a.bias ? a.bias[m] : 0.f), a.act, a.act_a, a.act_b);
      }
    }
  }
}

// z [rows, 2 I]: first | second -> (clamp(first) + 1) g sigmoid(alpha g), g = min(second, limit)
__global__ void __launch_bounds__(256)
clamped_glu_kernel(const float* __restrict__ z, float* __restrict__ out, long long total, int I,
                   float limit, float alpha) {
  US_PDL_PROLOGUE();
  const long long e = (long long)blockIdx.x * 256 + threadIdx.x;
  if (e >= total) return;
  const long long r = e / I;
  const float* row = z + r * 2 * I + (e - r * I);
  const float g = fminf(row[I], limit), u = fminf(fmaxf(row[0], -limit), limit);
  out[e] = (u + 1.f) * (g / (1.f + expf(-alpha * g)));
}

}  // namespace

US_API int us_clamped_glu_f32(const float* z, float* out, int rows, int I, float limit, float alpha,
                              void* stream_) {
  US_REQUIRE(z && out && rows >= 0 && I >= 1);
  const long long total = (long long)rows * I;
  if (total == 0) return US_OK;
  US_CUDA_CHECK(us::launch_pdl(clamped_glu_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0,
                               (cudaStream_t)stream_, z, out, total, I, limit, alpha));
  return US_OK;
}

// Same operand conventions as us_gemm_wx; act: 0 none, 3 gelu (erf), 5 square of relu, 6 xIELU (act_a,
// act_b).
US_API int us_gemm_f32(const float* W, const float* X, float* out, int G, int w_rows, int M, int K,
                       int x_rows, long long ldw, long long ldx, long long ldo, int act,
                       float act_a, float act_b, const float* bias, const int* tile_group, const int* tile_row0,
                       const int* tile_rows, const int* num_tiles, int max_tiles, void* stream_) {
  US_REQUIRE(W && X && out && G >= 1 && M >= 1 && K >= 1 && x_rows >= 0 &&
             (act == 0 || act == 3 || act == 5 || act == 6));
  US_REQUIRE(!num_tiles || (tile_group && tile_row0 && tile_rows && max_tiles >= 1 && !bias));
  if (x_rows == 0) return US_OK;
  const int tiles = num_tiles ? max_tiles : (x_rows + kT - 1) / kT;
  US_REQUIRE(tiles <= 65535);
  F32Args a{W, X, bias, out, ldw, ldx, ldo, w_rows, M, K, x_rows, act, tile_group, tile_row0,
            tile_rows, num_tiles, act_a, act_b};
  US_CUDA_CHECK(us::launch_pdl(gemm_f32_kernel, dim3((M + kT - 1) / kT, tiles), dim3(256), 0,
                               (cudaStream_t)stream_, a));
  return US_OK;
}
