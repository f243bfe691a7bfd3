// Latent attention over cache pages: a cached token is one normed latent c [R] and one rotated key
// part kr [RD] shared by all heads; queries arrive with W_uk folded in (ql = W_uk^T q, [R] per
// head) beside their rotated part, and the output is a mixture of latents (W_uv follows):
//
//   s_h(i, j) = scale (ql_h(i) . c_j + qr_h(i) . kr_j),   j <= i, i - j < window (0: no limit)
//   o_h(i)    = sum_j softmax_j(s_h(i, j)) c_j
//
//   us_latent_prep              norms of the query and key latents, rotation of the key part, pages
//   us_rotate_heads             rotation of the queries' rotated parts, in place
//   us_head_linear              a product per head: out[t, h] = W_h x[t, h], also times sigmoid(gate[t, h])
//   us_latent_attention_rows    any sizes, bf16 or FP32: one CTA per (query row, up to 16 heads)
//
// Channel 2i turns with channel 2i + 1 or, in halves, i with i + pairs; cosine and sine carry a factor.
// The angle is formed and reduced to a fraction of a turn in
// FP64, so far positions lose nothing before the FP32 sine and cosine.
#include "include/us_common.cuh"
#include "include/us_mma.cuh"
#include "include/us_tc05.cuh"

namespace {

__device__ __forceinline__ float ld1(const void* base, long long i, int bf16) {
  return bf16 ? us::bf2f(reinterpret_cast<const __nv_bfloat16*>(base)[i])
              : reinterpret_cast<const float*>(base)[i];
}
__device__ __forceinline__ void st1(void* base, long long i, int bf16, float v) {
  if (bf16) reinterpret_cast<__nv_bfloat16*>(base)[i] = us::f2bf(v);
  else reinterpret_cast<float*>(base)[i] = v;
}
__device__ __forceinline__ int seq_of(const int* cu, int B, int t) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

__device__ __forceinline__ void turn(int pos, double freq, float& c, float& s) {
  const double x = (double)pos * freq * 0.15915494309189535;      // turns
  sincospif(2.f * (float)(x - rint(x)), &s, &c);
}

constexpr int kPrepThreads = 128;

struct LatentPrep {
  void* x;
  long long ldx;
  int off_q, off_c, off_r, nq, nc, nr, pairs;
  const float *wq, *wc;
  const double* freq;
  const int *pos, *slots;
  void *cpages, *rpages;
  int ldc, ldr;
  float eps;
  int bf16;
  float mag;
  int halves;
};

__global__ void __launch_bounds__(kPrepThreads) latent_prep_kernel(const LatentPrep a) {
  US_PDL_PROLOGUE();
  __shared__ float2 part[kPrepThreads / 32];
  const int t = blockIdx.x, tid = threadIdx.x;
  const long long base = (long long)t * a.ldx;
  const long long slot = a.slots[t];
  float sq = 0.f, sc = 0.f;
  for (int c = tid; c < a.nq; c += kPrepThreads) {
    const float v = ld1(a.x, base + a.off_q + c, a.bf16);
    sq += v * v;
  }
  for (int c = tid; c < a.nc; c += kPrepThreads) {
    const float v = ld1(a.x, base + a.off_c + c, a.bf16);
    sc += v * v;
  }
  sq = us::warp_sum(sq);
  sc = us::warp_sum(sc);
  if ((tid & 31) == 0) part[tid >> 5] = make_float2(sq, sc);
  __syncthreads();
  sq = sc = 0.f;
#pragma unroll
  for (int w = 0; w < kPrepThreads / 32; ++w) {
    sq += part[w].x;
    sc += part[w].y;
  }
  const float iq = 1.f / sqrtf(sq / (float)a.nq + a.eps), ic = 1.f / sqrtf(sc / (float)a.nc + a.eps);
  for (int c = tid; c < a.nq; c += kPrepThreads)
    st1(a.x, base + a.off_q + c, a.bf16, ld1(a.x, base + a.off_q + c, a.bf16) * iq * a.wq[c]);
  if (slot < 0) return;
  for (int c = tid; c < a.nc; c += kPrepThreads)
    st1(a.cpages, slot * a.ldc + c, a.bf16, ld1(a.x, base + a.off_c + c, a.bf16) * ic * a.wc[c]);
  const int pos = a.pos[t];
  const long long from = base + a.off_r, to = slot * a.ldr;
  for (int i = tid; i < a.pairs; i += kPrepThreads) {
    const int p = a.halves ? i : 2 * i, q = a.halves ? i + a.pairs : 2 * i + 1;
    const float u = ld1(a.x, from + p, a.bf16), v = ld1(a.x, from + q, a.bf16);
    float c, s;
    turn(pos, a.freq[i], c, s);
    c *= a.mag;
    s *= a.mag;
    st1(a.rpages, to + p, a.bf16, u * c - v * s);
    st1(a.rpages, to + q, a.bf16, v * c + u * s);
  }
  for (int i = 2 * a.pairs + tid; i < a.nr; i += kPrepThreads)
    st1(a.rpages, to + i, a.bf16, ld1(a.x, from + i, a.bf16));
}

// x [T, ldx]: head h's pairs start at column off + h * hs.  A thread per (pair, group of heads).
__global__ void __launch_bounds__(256)
rotate_heads_kernel(void* __restrict__ x, long long ldx, int off, int hs, int H,
                    const double* __restrict__ freq, int pairs, const int* __restrict__ pos,
                    long long total, int bf16, float mag, int halves) {
  US_PDL_PROLOGUE();
  const long long e = (long long)blockIdx.x * 256 + threadIdx.x;
  if (e >= total) return;
  const int groups = (H + 3) / 4;
  const int i = (int)(e % pairs);
  const long long r = e / pairs;
  const int h0 = (int)(r % groups) * 4;
  const long long t = r / groups;
  float c, s;
  turn(pos[t], freq[i], c, s);
  c *= mag;
  s *= mag;
  const int p = halves ? i : 2 * i, gap = halves ? pairs : 1;
  for (int h = h0; h < min(H, h0 + 4); ++h) {
    const long long at = t * ldx + off + (long long)h * hs + p;
    const float u = ld1(x, at, bf16), v = ld1(x, at + gap, bf16);
    st1(x, at, bf16, u * c - v * s);
    st1(x, at + gap, bf16, v * c + u * s);
  }
}

// ---------------------------------------------------------- products per head --
struct HeadLinear {
  const void *W, *X;          // W [H, M, K] (rows at ldw, heads at hsw), X rows at ldx, heads at hsx
  void* out;
  long long hsw, ldw, ldx, hsx, ldo, hso;
  int H, M, K, rows;
  const void* gate;           // or null: feature m of head h at column h M + m, rows at ldg
  long long ldg;
  const int* gate_rows;       // row of `gate` for every row of X, or null: the same
};

__device__ __forceinline__ float gated(const HeadLinear& a, float v, int h, int r, int m, int bf16) {
  if (!a.gate) return v;
  const long long row = a.gate_rows ? a.gate_rows[r] : r;
  return v / (1.f + expf(-ld1(a.gate, row * a.ldg + (long long)h * a.M + m, bf16)));
}

__global__ void __launch_bounds__(256) head_linear_f32_kernel(const HeadLinear a) {
  US_PDL_PROLOGUE();
  constexpr int kT = 64, kK = 16;
  __shared__ float xs[kK][kT + 4], ws[kK][kT + 4];
  const int h = blockIdx.z, r0 = blockIdx.y * kT, m0 = blockIdx.x * kT;
  const float* W = (const float*)a.W + h * a.hsw;
  const float* X = (const float*)a.X + h * a.hsx;
  float* out = (float*)a.out + h * a.hso;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += kK) {
    for (int e = threadIdx.x; e < kT * kK; e += 256) {
      const int i = e / kK, k = e - i * kK;
      const bool kin = k0 + k < a.K;
      xs[k][i] = (kin && r0 + i < a.rows) ? X[(long long)(r0 + i) * a.ldx + k0 + k] : 0.f;
      ws[k][i] = (kin && m0 + i < a.M) ? W[(long long)(m0 + i) * a.ldw + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kK; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xs[k][ty * 4 + i], ws[k][tx * 4 + j], acc[i][j]);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (r0 + ty * 4 + i < a.rows && m0 + tx * 4 + j < a.M)
        out[(long long)(r0 + ty * 4 + i) * a.ldo + m0 + tx * 4 + j] =
            gated(a, acc[i][j], h, r0 + ty * 4 + i, m0 + tx * 4 + j, 0);
}

// 64 rows x 64 features of one head; a warp takes 16 rows.  K in steps of 64, the next step's
// tiles on their way (cp.async) while one multiplies.
__global__ void __launch_bounds__(128) head_linear_kernel(const HeadLinear a) {
  US_PDL_PROLOGUE();
  __shared__ __align__(1024) uint8_t sm[2][2][64 * 128];
  const int h = blockIdx.z, r0 = blockIdx.y * 64, m0 = blockIdx.x * 64;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lrow = lane & 15, lhalf = lane >> 4;
  const __nv_bfloat16* W = (const __nv_bfloat16*)a.W + h * a.hsw;
  const __nv_bfloat16* X = (const __nv_bfloat16*)a.X + h * a.hsx;
  auto fetch = [&](int k0, int buf) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (tid >> 3) + i * 16, c = tid & 7, k = k0 + c * 8;
      const uint32_t dx = tc::smem_u32(sm[buf][0]) + us::swz(r, c, 8), dw = tc::smem_u32(sm[buf][1]) + us::swz(r, c, 8);
      if (r0 + r < a.rows && k < a.K) us::cp16(dx, X + (long long)(r0 + r) * a.ldx + k);
      else us::zero16(dx);
      if (m0 + r < a.M && k < a.K) us::cp16(dw, W + (long long)(m0 + r) * a.ldw + k);
      else us::zero16(dw);
    }
    us::cp_commit();
  };
  float acc[8][4] = {};
  fetch(0, 0);
  int buf = 0;
  for (int k0 = 0; k0 < a.K; k0 += 64, buf ^= 1) {
    us::cp_wait<0>();
    __syncthreads();
    if (k0 + 64 < a.K) fetch(k0 + 64, buf ^ 1);
    const uint32_t sx = tc::smem_u32(sm[buf][0]), sw = tc::smem_u32(sm[buf][1]);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      uint32_t x[4];
      us::ldsm4(x, sx + us::swz(warp * 16 + lrow, 2 * k + lhalf, 8));
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        uint32_t w[4];
        us::ldsm4(w, sw + us::swz(n * 16 + lrow, 2 * k + lhalf, 8));
        us::mma16816(acc[2 * n], x[0], x[1], x[2], x[3], w[0], w[2]);
        us::mma16816(acc[2 * n + 1], x[0], x[1], x[2], x[3], w[1], w[3]);
      }
    }
  }
  __nv_bfloat16* out = (__nv_bfloat16*)a.out + h * a.hso;
  const bool pairs = ((a.ldo | a.hso) & 1) == 0;
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = r0 + warp * 16 + (lane >> 2) + e * 8, m = m0 + n * 8 + (lane & 3) * 2;
      if (r >= a.rows || m >= a.M) continue;
      __nv_bfloat16* o = out + (long long)r * a.ldo + m;
      const bool both = m + 1 < a.M;
      const float v0 = gated(a, acc[n][e * 2], h, r, m, 1), v1 = both ? gated(a, acc[n][e * 2 + 1], h, r, m + 1, 1) : 0.f;
      if (pairs && both) {
        *reinterpret_cast<__nv_bfloat162*>(o) = __floats2bfloat162_rn(v0, v1);
      } else {
        o[0] = us::f2bf(v0);
        if (both) o[1] = us::f2bf(v1);
      }
    }
}

// ---------------------------------------------------------------- row form --
struct LatentAttn {
  const void *ql, *qr;        // [T, H, R] and [T, H, RD]: rows at ld, heads at hs
  long long ldql, ldqr;
  int hsql, hsqr;
  const void *cp, *rp;        // pages [n, page, ldc], [n, page, ldr]
  int ldc, ldr;
  void* out;                  // [T, H, ...]: columns R .. hso of a head are zeroed
  long long ldo;
  int hso;
  const int *cu, *pos, *seq_lens, *page_table;
  int T, B, H, R, RD, page, max_pages, window, bf16, per;
  float scale;
};

constexpr int kRowThreads = 256;
constexpr int kRowKeys = 16;

__global__ void __launch_bounds__(kRowThreads) latent_rows_kernel(const LatentAttn a) {
  US_PDL_PROLOGUE();
  extern __shared__ __align__(16) float smf[];
  const int D = a.R + a.RD, ldk = D | 1, R = a.R;
  const int h0 = blockIdx.y * a.per, nh = min(a.per, a.H - h0);
  float* qs = smf;                         // [per][D], scaled
  float* ks = qs + a.per * D;              // [kRowKeys][ldk]
  float* os = ks + kRowKeys * ldk;         // [per][R]
  float* ps = os + a.per * R;              // [per][kRowKeys]
  float* mx = ps + a.per * kRowKeys;       // [per] each
  float* sum = mx + a.per;
  float* fac = sum + a.per;
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int s = seq_of(a.cu, a.B, t);
  const bool live = !a.seq_lens || a.seq_lens[s] > 0;
  for (int e = tid; e < nh * D; e += kRowThreads) {
    const int h = e / D, d = e - h * D;
    const float v = d < R ? ld1(a.ql, t * a.ldql + (long long)(h0 + h) * a.hsql + d, a.bf16)
                          : ld1(a.qr, t * a.ldqr + (long long)(h0 + h) * a.hsqr + d - R, a.bf16);
    qs[e] = live ? v * a.scale : 0.f;
  }
  for (int e = tid; e < nh; e += kRowThreads) { mx[e] = -INFINITY; sum[e] = 0.f; }
  for (int e = tid; e < nh * R; e += kRowThreads) os[e] = 0.f;
  const int i = live ? a.pos[t] : -1;
  const int lo = a.window > 0 ? max(0, i - a.window + 1) : 0;
  const int* pt = a.page_table + (long long)s * a.max_pages;
  for (int j0 = lo; j0 <= i; j0 += kRowKeys) {
    const int nj = min(kRowKeys, i - j0 + 1);
    __syncthreads();
    for (int e = tid; e < nj * D; e += kRowThreads) {
      const int j = e / D, d = e - j * D, key = j0 + j;
      const long long at = (long long)pt[key / a.page] * a.page + key % a.page;
      ks[j * ldk + d] = d < R ? ld1(a.cp, at * a.ldc + d, a.bf16) : ld1(a.rp, at * a.ldr + d - R, a.bf16);
    }
    __syncthreads();
    for (int e = tid; e < nh * kRowKeys; e += kRowThreads) {
      const int h = e / kRowKeys, j = e - h * kRowKeys;
      float d = 0.f;
      if (j < nj)
        for (int x = 0; x < D; ++x) d = fmaf(qs[h * D + x], ks[j * ldk + x], d);
      ps[e] = j < nj ? d : -INFINITY;
    }
    __syncthreads();
    for (int h = warp; h < nh; h += kRowThreads / 32) {
      const float sc = lane < kRowKeys ? ps[h * kRowKeys + lane] : -INFINITY;
      const float m0 = mx[h], m = fmaxf(m0, us::warp_max(sc));
      const float p = lane < nj ? expf(sc - m) : 0.f;
      const float add = us::warp_sum(p);
      if (lane < kRowKeys) ps[h * kRowKeys + lane] = p;
      if (lane == 0) {
        fac[h] = expf(m0 - m);
        sum[h] = sum[h] * fac[h] + add;
        mx[h] = m;
      }
    }
    __syncthreads();
    for (int e = tid; e < nh * R; e += kRowThreads) {
      const int h = e / R, c = e - h * R;
      float acc = os[e] * fac[h];
      for (int j = 0; j < nj; ++j) acc = fmaf(ps[h * kRowKeys + j], ks[j * ldk + c], acc);
      os[e] = acc;
    }
  }
  __syncthreads();
  for (int e = tid; e < nh * a.hso; e += kRowThreads) {
    const int h = e / a.hso, c = e - h * a.hso;
    st1(a.out, t * a.ldo + (long long)(h0 + h) * a.hso + c, a.bf16,
        c < R && live ? os[h * R + c] / sum[h] : 0.f);
  }
}

}  // namespace

US_API int us_latent_prep(void* x, long long ldx, int off_q, int off_c, int off_r, int nq, int nc,
                          int nr, const float* wq, const float* wc, const double* freq, int pairs,
                          const int* pos, const int* slots, void* cpages, int ldc, void* rpages,
                          int ldr, int T, float eps, float mag, int halves, int bf16, void* stream_) {
  US_REQUIRE(x && wq && wc && pos && slots && cpages && rpages && T >= 0 && nq >= 1 && nc >= 1 &&
             nr >= 0 && ldc >= nc && ldr >= nr && 2 * pairs <= nr && (pairs == 0 || freq));
  if (T == 0) return US_OK;
  LatentPrep a{x, ldx, off_q, off_c, off_r, nq, nc, nr, pairs, wq, wc, freq, pos, slots, cpages,
               rpages, ldc, ldr, eps, bf16, mag, halves};
  US_CUDA_CHECK(us::launch_pdl(latent_prep_kernel, dim3(T), dim3(kPrepThreads), 0,
                               (cudaStream_t)stream_, a));
  return US_OK;
}

US_API int us_rotate_heads(void* x, long long ldx, int off, int hs, int H, const double* freq,
                           int pairs, const int* pos, int T, float mag, int halves, int bf16,
                           void* stream_) {
  US_REQUIRE(x && freq && pos && T >= 0 && H >= 1 && pairs >= 1);
  const long long total = (long long)T * ((H + 3) / 4) * pairs;
  if (total == 0) return US_OK;
  US_CUDA_CHECK(us::launch_pdl(rotate_heads_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0,
                               (cudaStream_t)stream_, x, ldx, off, hs, H, freq, pairs, pos, total, bf16, mag, halves));
  return US_OK;
}

// gate (or null) [.., H M] rows at ldg: the result times its sigmoid; gate_rows (or null): its row for every
// row of X.
US_API int us_head_linear(const void* W, const void* X, void* out, long long hsw, long long ldw,
                          long long ldx, long long hsx, long long ldo, long long hso, int H, int M,
                          int K, int rows, const void* gate, long long ldg, const int* gate_rows,
                          int bf16, void* stream_) {
  US_REQUIRE(W && X && out && H >= 1 && M >= 1 && K >= 1 && rows >= 0 && H <= 65535);
  if (rows == 0) return US_OK;
  HeadLinear a{W, X, out, hsw, ldw, ldx, hsx, ldo, hso, H, M, K, rows, gate, ldg, gate_rows};
  const dim3 grid(us::ceil_div(M, 64), us::ceil_div(rows, 64), H);
  if (bf16) {
    US_REQUIRE((K % 8) == 0 && (ldw % 8) == 0 && (hsw % 8) == 0 && (ldx % 8) == 0 && (hsx % 8) == 0 &&
               ((uintptr_t)W % 16) == 0 && ((uintptr_t)X % 16) == 0);
    US_CUDA_CHECK(us::launch_pdl(head_linear_kernel, grid, dim3(128), 0, (cudaStream_t)stream_, a));
  } else {
    US_CUDA_CHECK(us::launch_pdl(head_linear_f32_kernel, grid, dim3(256), 0, (cudaStream_t)stream_, a));
  }
  return US_OK;
}

// Attention of T rows (rows of sequence s at cu[s] .. cu[s + 1], keys up to a row's own position).
US_API int us_latent_attention_rows(const void* ql, long long ldql, int hsql, const void* qr,
                                    long long ldqr, int hsqr, const void* cpages, int ldc,
                                    const void* rpages, int ldr, void* out, long long ldo, int hso,
                                    const int* cu, const int* pos, const int* seq_lens,
                                    const int* page_table, int T, int B, int H, int R, int RD,
                                    int page, int max_pages, int window, float scale, int bf16,
                                    void* stream_) {
  US_REQUIRE(ql && qr && cpages && rpages && out && cu && pos && page_table && T >= 0 && B >= 1 &&
             H >= 1 && R >= 1 && RD >= 0 && page >= 1 && hso >= R && ldc >= R && ldr >= RD);
  if (T == 0) return US_OK;
  const int D = R + RD;
  constexpr size_t kMost = 220 * 1024;
  auto bytes = [&](int per) {
    return 4 * ((size_t)per * (D + R + kRowKeys + 3) + (size_t)kRowKeys * (D | 1));
  };
  int per = min(16, H);
  while (per > 1 && bytes(per) > kMost) per /= 2;
  if (bytes(per) > kMost) return US_ERR_LIMIT;
  LatentAttn a{ql, qr, ldql, ldqr, hsql, hsqr, cpages, rpages, ldc, ldr, out, ldo, hso, cu, pos,
               seq_lens, page_table, T, B, H, R, RD, page, max_pages, window, bf16, per, scale};
  static bool configured = false;
  if (!configured) {
    US_CUDA_CHECK(cudaFuncSetAttribute(latent_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                       (int)kMost));
    configured = true;
  }
  US_CUDA_CHECK(us::launch_pdl(latent_rows_kernel, dim3(T, us::ceil_div(H, per)), dim3(kRowThreads),
                               bytes(per), (cudaStream_t)stream_, a));
  return US_OK;
}
