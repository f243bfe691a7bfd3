// Row operators of decoders that norm a sublayer's *output* before it joins the FP32 residual:
//
//   embed_rows         residual = FP32 row of the table, x = the same row in the model's type
//   output_norm_add    y = sublayer output, or w * sum of routed expert rows
//                          + sigmoid(residual . gate) * shared expert row
//                      residual += y / rms(y) * gain;  x = residual in the model's type, or
//                      residual / rms(residual) * final_gain when the layer is the last one
//   row_norm_kv        q and k normalised over their whole projection row (all heads at once),
//                      q left in place, k and v written to the cache pages
//   table_route_sort   experts looked up by token id, routes sorted by expert (see moe_route.cu)
//
// Rows are padded to a multiple of 8 columns with zeros; `width` is the true column count that
// means divide by.  Element types: 1 = bf16, 0 = fp32.  All arithmetic is FP32.
#include "include/us_common.cuh"

namespace {

constexpr int kThreads = 256;

__device__ __forceinline__ float4 ld4(const void* base, long long i, int bf16) {
  if (bf16) {
    us::Pack8 p;
    p.u = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(base) + i);
    return make_float4(us::bf2f(p.b[0]), us::bf2f(p.b[1]), us::bf2f(p.b[2]), us::bf2f(p.b[3]));
  }
  return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(base) + i);
}
__device__ __forceinline__ void st4(void* base, long long i, int bf16, float4 v) {
  if (bf16) {
    us::Pack8 p;
    p.b[0] = us::f2bf(v.x); p.b[1] = us::f2bf(v.y); p.b[2] = us::f2bf(v.z); p.b[3] = us::f2bf(v.w);
    *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(base) + i) = p.u;
  } else {
    *reinterpret_cast<float4*>(reinterpret_cast<float*>(base) + i) = v;
  }
}
__device__ __forceinline__ float ld1(const void* base, long long i, int bf16) {
  return bf16 ? us::bf2f(reinterpret_cast<const __nv_bfloat16*>(base)[i])
              : reinterpret_cast<const float*>(base)[i];
}
__device__ __forceinline__ void st1(void* base, long long i, int bf16, float v) {
  if (bf16) reinterpret_cast<__nv_bfloat16*>(base)[i] = us::f2bf(v);
  else reinterpret_cast<float*>(base)[i] = v;
}
__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

__global__ void __launch_bounds__(kThreads)
embed_rows_kernel(const int* __restrict__ ids, const void* __restrict__ table,
                  float* __restrict__ residual, void* __restrict__ x, int W, int vocab, int bf16,
                  unsigned int* status) {
  US_PDL_PROLOGUE();
  const int t = blockIdx.x, id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0) us_dev_fail(status, US_DEV_BOUNDS);
  for (int c = threadIdx.x * 4; c < W; c += kThreads * 4) {
    const float4 v = ok ? ld4(table, (long long)id * W + c, bf16) : make_float4(0.f, 0.f, 0.f, 0.f);
    *reinterpret_cast<float4*>(residual + (long long)t * W + c) = v;
    st4(x, (long long)t * W + c, bf16, v);
  }
}

struct OutNormArgs {
  const void* y;              // [T, W] sublayer output, or null: routed rows
  const void* y_perm;         // [R, W] expert rows
  const int* perm;            // [T, top] row of each route
  float route_w;
  int top;
  const void* shared;         // [T, W] or null
  const float* shared_gate;   // [W] or null (no gate: added as it is)
  float* residual;            // [T, W]
  void* x;                    // [T, W]
  float gain, final_gain, eps;
  int W, width, bf16, last;
};

__global__ void __launch_bounds__(kThreads) output_norm_add_kernel(const OutNormArgs a) {
  US_PDL_PROLOGUE();
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[33];
  const long long base = (long long)blockIdx.x * a.W;
  const int W = a.W;
  float sg = 1.f;
  if (a.shared && a.shared_gate) {
    float d = 0.f;
    for (int c = threadIdx.x * 4; c < W; c += kThreads * 4) {
      const float4 r = *reinterpret_cast<const float4*>(a.residual + base + c);
      const float4 w = *reinterpret_cast<const float4*>(a.shared_gate + c);
      d += r.x * w.x + r.y * w.y + r.z * w.z + r.w * w.w;
    }
    d = us::block_sum(d, scratch);
    sg = 1.f / (1.f + expf(-d));
  }
  float ss = 0.f;
  for (int c = threadIdx.x * 4; c < W; c += kThreads * 4) {
    float4 v;
    if (a.y) {
      v = ld4(a.y, base + c, a.bf16);
    } else {
      v = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int k = 0; k < a.top; ++k) {
        const long long r = a.perm[(long long)blockIdx.x * a.top + k];
        const float4 e = ld4(a.y_perm, r * W + c, a.bf16);
        v.x += e.x; v.y += e.y; v.z += e.z; v.w += e.w;
      }
      v.x *= a.route_w; v.y *= a.route_w; v.z *= a.route_w; v.w *= a.route_w;
    }
    if (a.shared) {
      const float4 e = ld4(a.shared, base + c, a.bf16);
      v.x += sg * e.x; v.y += sg * e.y; v.z += sg * e.z; v.w += sg * e.w;
    }
    *reinterpret_cast<float4*>(row + c) = v;
    ss += sq4(v);
  }
  ss = us::block_sum(ss, scratch);
  const float m = a.gain / sqrtf(ss / (float)a.width + a.eps);
  float s2 = 0.f;
  for (int c = threadIdx.x * 4; c < W; c += kThreads * 4) {
    const float4 v = *reinterpret_cast<const float4*>(row + c);
    float4 r = *reinterpret_cast<const float4*>(a.residual + base + c);
    r.x += v.x * m; r.y += v.y * m; r.z += v.z * m; r.w += v.w * m;
    *reinterpret_cast<float4*>(a.residual + base + c) = r;
    if (a.last) {
      *reinterpret_cast<float4*>(row + c) = r;
      s2 += sq4(r);
    } else {
      st4(a.x, base + c, a.bf16, r);
    }
  }
  if (!a.last) return;
  s2 = us::block_sum(s2, scratch);
  const float f = a.final_gain / sqrtf(s2 / (float)a.width + a.eps);
  for (int c = threadIdx.x * 4; c < W; c += kThreads * 4) {
    float4 r = *reinterpret_cast<const float4*>(row + c);
    r.x *= f; r.y *= f; r.z *= f; r.w *= f;
    st4(a.x, base + c, a.bf16, r);
  }
}

struct RowNormKv {
  void* x;                    // projection rows (q normalised in place)
  long long ldx;
  int off_q, off_k, off_v, nq, nk, nv;   // nk = 0: the layer has no keys of its own
  const float *wq, *wk;
  const int* slots;           // cache slot of every row, negative: not written
  void *kc, *vc;              // [slots, nk], [slots, nv]
  float eps;
  int bf16;
};

// Both sums in one pass over the row and one exchange.  VEC: every width is a multiple of 4.
template <bool VEC>
__global__ void __launch_bounds__(kThreads) row_norm_kv_kernel(const RowNormKv a) {
  US_PDL_PROLOGUE();
  constexpr int U = VEC ? 4 : 1;
  __shared__ float2 part[kThreads / 32];
  const long long base = (long long)blockIdx.x * a.ldx;
  const int tid = threadIdx.x;
  auto load = [&](long long i) -> float4 {
    return VEC ? ld4(a.x, base + i, a.bf16) : make_float4(ld1(a.x, base + i, a.bf16), 0.f, 0.f, 0.f);
  };
  auto weight = [&](const float* w, int c) -> float4 {
    return VEC ? *reinterpret_cast<const float4*>(w + c) : make_float4(w[c], 0.f, 0.f, 0.f);
  };
  auto store = [&](void* dst, long long i, float4 v) {
    if (VEC) st4(dst, i, a.bf16, v);
    else st1(dst, i, a.bf16, v.x);
  };
  const long long slot = a.nk ? a.slots[blockIdx.x] : -1;
  float sq = 0.f, sk = 0.f;
  for (int c = tid * U; c < a.nq; c += kThreads * U) sq += sq4(load(a.off_q + c));
  for (int c = tid * U; c < a.nk; c += kThreads * U) sk += sq4(load(a.off_k + c));
  sq = us::warp_sum(sq);
  sk = us::warp_sum(sk);
  if ((tid & 31) == 0) part[tid >> 5] = make_float2(sq, sk);
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < kThreads / 32; ++w) {
    sq += part[w].x;
    sk += part[w].y;
  }
  const float iq = 1.f / sqrtf(sq / (float)a.nq + a.eps);
  for (int c = tid * U; c < a.nq; c += kThreads * U) {
    float4 v = load(a.off_q + c);
    const float4 w = weight(a.wq, c);
    v.x *= iq * w.x; v.y *= iq * w.y; v.z *= iq * w.z; v.w *= iq * w.w;
    store(a.x, base + a.off_q + c, v);
  }
  if (slot < 0) return;
  const float ik = 1.f / sqrtf(sk / (float)a.nk + a.eps);
  for (int c = tid * U; c < a.nk; c += kThreads * U) {
    float4 v = load(a.off_k + c);
    const float4 w = weight(a.wk, c);
    v.x *= ik * w.x; v.y *= ik * w.y; v.z *= ik * w.z; v.w *= ik * w.w;
    store(a.kc, slot * a.nk + c, v);
  }
  for (int c = tid * U; c < a.nv; c += kThreads * U) store(a.vc, slot * a.nv + c, load(a.off_v + c));
}

// tanh over a column range of the rows, in place.
__global__ void __launch_bounds__(kThreads)
tanh_cols_kernel(void* __restrict__ x, long long ldx, int off, int n, int rows, int bf16) {
  US_PDL_PROLOGUE();
  const long long e = (long long)blockIdx.x * kThreads + threadIdx.x;
  if (e >= (long long)rows * n) return;
  const long long t = e / n, i = t * ldx + off + (e - t * n);
  st1(x, i, bf16, tanhf(ld1(x, i, bf16)));
}

}  // namespace

US_API int us_embed_rows(const int* ids, const void* table, float* residual, void* x, int T, int W,
                         int vocab, int bf16, void* stream_) {
  US_REQUIRE(ids && table && residual && x && T >= 0 && W >= 8 && (W % 8) == 0);
  if (T == 0) return US_OK;
  US_CUDA_CHECK(us::launch_pdl(embed_rows_kernel, dim3(T), dim3(kThreads), 0, (cudaStream_t)stream_,
                               ids, table, residual, x, W, vocab, bf16, us_status_ptr()));
  return US_OK;
}

US_API int us_output_norm_add(const void* y, const void* y_perm, const int* perm, float route_w,
                              int top, const void* shared, const float* shared_gate,
                              float* residual, void* x, float gain, float final_gain, int last,
                              int T, int W, int width, float eps, int bf16, void* stream_) {
  US_REQUIRE((y || (y_perm && perm && top >= 1)) && residual && x && T >= 0 && W >= 8 &&
             (W % 8) == 0 && width >= 1 && width <= W);
  if (W > 32768) return US_ERR_LIMIT;
  if (T == 0) return US_OK;
  OutNormArgs a{y, y_perm, perm, route_w, top, shared, shared_gate, residual, x, gain, final_gain,
                eps, W, width, bf16, last};
  const size_t smem = (size_t)W * sizeof(float);
  static bool configured = false;
  if (!configured) {
    US_CUDA_CHECK(cudaFuncSetAttribute(output_norm_add_kernel,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024));
    configured = true;
  }
  US_CUDA_CHECK(us::launch_pdl(output_norm_add_kernel, dim3(T), dim3(kThreads), smem,
                               (cudaStream_t)stream_, a));
  return US_OK;
}

US_API int us_row_norm_kv(void* x, long long ldx, int off_q, int off_k, int off_v, int nq, int nk,
                          int nv, const float* wq, const float* wk, const int* slots, void* kc,
                          void* vc, int T, float eps, int bf16, void* stream_) {
  US_REQUIRE(x && wq && T >= 0 && nq >= 1);
  US_REQUIRE(nk == 0 || (nv >= 1 && wk && slots && kc && vc));
  if (T == 0) return US_OK;
  RowNormKv a{x, ldx, off_q, off_k, off_v, nq, nk, nv, wq, wk, slots, kc, vc, eps, bf16};
  const bool vec = ((nq | nk | nv | off_q | off_k | off_v) & 3) == 0 && (ldx & 3) == 0 &&
                   (((uintptr_t)x | (uintptr_t)kc | (uintptr_t)vc | (uintptr_t)wq | (uintptr_t)wk) % 16) == 0;
  US_CUDA_CHECK(us::launch_pdl(vec ? row_norm_kv_kernel<true> : row_norm_kv_kernel<false>, dim3(T),
                               dim3(kThreads), 0, (cudaStream_t)stream_, a));
  return US_OK;
}

US_API int us_tanh_cols(void* x, long long ldx, int off, int n, int rows, int bf16, void* stream_) {
  US_REQUIRE(x && n >= 1 && rows >= 0 && off >= 0);
  if (rows == 0) return US_OK;
  const long long total = (long long)rows * n;
  US_CUDA_CHECK(us::launch_pdl(tanh_cols_kernel, dim3((unsigned)((total + kThreads - 1) / kThreads)),
                               dim3(kThreads), 0, (cudaStream_t)stream_, x, ldx, off, n, rows, bf16));
  return US_OK;
}
