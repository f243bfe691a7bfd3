// Causal attention over cache pages whose heads share their softmax weights:
//
//   p_g(i, j) = softmax_j(scale q_g(i) . k(j))       over the keys i sees
//   w_h(i, j) = sum_g T[h, g] p_g(i, j)
//   o_h(i)    = sum_j w_h(i, j) v_{kv(h)}(j)
//
// Query i sees key j <= i inside a window (i - j < size) or among the first `keep` keys of the
// sequence; both limits are off when not positive.  The mixture needs every head's *normalised*
// weight of a key before any head's value product, so the softmax statistics (maximum and sum
// per head) of all heads come first and the scores are formed a second time for the product.
//
// General form (any head width, bf16 or FP32 pages): one CTA per query row, all heads.  Keys
// are read through the page table, the key list of a query being its kept keys followed by its
// window.  All arithmetic is FP32.
#include "include/us_common.cuh"

namespace {

constexpr int kTile = 32;
constexpr int kThreads = 256;

struct MixArgs {
  const void* q;              // [rows, H * D] rows at ldq
  const void *kc, *vc;        // [pages, page, G, D], [pages, page, G, V]
  const float* talk;          // [H, H]
  void* out;                  // [rows, ldo]
  const int *cu, *pos, *page_table;
  long long ldq, ldo;
  int B, H, G, D, V, page, max_pages, size, keep, bf16;
  const int* seq_lens;        // decode: 0 marks a padding row
  float scale;
};

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

__global__ void __launch_bounds__(kThreads) head_mix_row_kernel(const MixArgs a) {
  US_PDL_PROLOGUE();
  extern __shared__ __align__(16) float sm[];
  const int H = a.H, G = a.G, D = a.D, V = a.V, rep = H / G;
  float* qs = sm;                      // [H, D], scaled
  float* ps = qs + H * D;              // [H, kTile] scores, then probabilities
  float* ws = ps + H * kTile;          // [H, kTile] mixed weights
  float* mx = ws + H * kTile;          // [H]
  float* sum = mx + H;                 // [H]
  float* os = sum + H;                 // [H, V]
  __shared__ long long where[kTile];   // cache slots of the tile's keys
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int s = seq_of(a.cu, a.B, t);
  const long long orow = (long long)t * a.ldo;
  if (a.seq_lens && a.seq_lens[s] <= 0) {
    for (int c = tid; c < a.ldo; c += kThreads) st1(a.out, orow + c, a.bf16, 0.f);
    return;
  }
  const int i = a.pos[t];
  const int lo = a.size > 0 ? max(0, i - a.size + 1) : 0;
  const int kept = min(max(a.keep, 0), lo);
  const int n = kept + i - lo + 1;
  for (int e = tid; e < H * D; e += kThreads)
    qs[e] = ld1(a.q, (long long)t * a.ldq + e, a.bf16) * a.scale;
  for (int e = tid; e < H; e += kThreads) { mx[e] = -INFINITY; sum[e] = 0.f; }
  for (int e = tid; e < H * V; e += kThreads) os[e] = 0.f;
  const int* pt = a.page_table + (long long)s * a.max_pages;
  for (int pass = 0; pass < 2; ++pass) {
    for (int j0 = 0; j0 < n; j0 += kTile) {
      const int nj = min(kTile, n - j0);
      __syncthreads();
      if (tid < nj) {
        const int x = j0 + tid, key = x < kept ? x : lo + x - kept;
        where[tid] = (long long)pt[key / a.page] * a.page + key % a.page;
      }
      __syncthreads();
      // scores: a warp takes a (key, kv head) pair, its lanes the channels
      for (int e = warp; e < nj * G; e += kThreads / 32) {
        const int j = e / G, u = e - j * G;
        const long long kb = (where[j] * G + u) * D;
        float kv[8];
#pragma unroll
        for (int x = 0; x < 8; ++x) kv[x] = x * 32 + lane < D ? ld1(a.kc, kb + x * 32 + lane, a.bf16) : 0.f;
        for (int r = 0; r < rep; ++r) {
          const float* q = qs + (u * rep + r) * D;
          float d = 0.f;
#pragma unroll
          for (int x = 0; x < 8; ++x)
            if (x * 32 + lane < D) d = fmaf(q[x * 32 + lane], kv[x], d);
          d = us::warp_sum(d);
          if (lane == 0) ps[(u * rep + r) * kTile + j] = d;
        }
      }
      __syncthreads();
      for (int h = warp; h < H; h += kThreads / 32) {
        const float sc = lane < nj ? ps[h * kTile + lane] : -INFINITY;
        if (pass == 0) {
          const float m = fmaxf(mx[h], us::warp_max(sc));
          const float add = us::warp_sum(lane < nj ? expf(sc - m) : 0.f);
          __syncwarp();
          if (lane == 0) {
            sum[h] = sum[h] * expf(mx[h] - m) + add;
            mx[h] = m;
          }
        } else {
          ps[h * kTile + lane] = lane < nj ? expf(sc - mx[h]) / sum[h] : 0.f;
        }
      }
      if (pass == 0) continue;
      __syncthreads();
      for (int e = tid; e < H * kTile; e += kThreads) {
        const int h = e / kTile, j = e - h * kTile;
        float w = 0.f;
        for (int g = 0; g < H; ++g) w = fmaf(a.talk[h * H + g], ps[g * kTile + j], w);
        ws[e] = w;
      }
      __syncthreads();
      for (int e = tid; e < H * V; e += kThreads) {
        const int h = e / V, c = e - h * V;
        float acc = os[e];
        for (int j = 0; j < nj; ++j)
          acc = fmaf(ws[h * kTile + j], ld1(a.vc, (where[j] * G + h / rep) * V + c, a.bf16), acc);
        os[e] = acc;
      }
    }
  }
  __syncthreads();
  for (int c = tid; c < a.ldo; c += kThreads)
    st1(a.out, orow + c, a.bf16, c < H * V ? os[c] : 0.f);
}

}  // namespace

// q [rows, H * D] (row stride ldq) of the packed sequences cu [B + 1], positions pos [rows];
// every key up to a row's own position is in the pages already.  Output rows are ldo wide
// (columns past H * V are zeroed).
US_API int us_head_mix_attention(const void* q, const void* kc, const void* vc, const float* talk,
                                 void* out, const int* cu, const int* pos, const int* page_table,
                                 const int* seq_lens, long long ldq, long long ldo, int rows, int B,
                                 int H, int G, int D, int V, int page, int max_pages, int size,
                                 int keep, float scale, int bf16, void* stream_) {
  US_REQUIRE(q && kc && vc && talk && out && cu && pos && page_table && rows >= 0 && B >= 1);
  US_REQUIRE(H >= 1 && G >= 1 && H % G == 0 && D >= 1 && V >= 1 && page >= 1 && max_pages >= 1 &&
             ldo >= (long long)H * V);
  if (D > 256) return US_ERR_UNSUPPORTED;
  if (rows == 0) return US_OK;
  const size_t smem = (size_t)(H * D + 2 * H * kTile + 2 * H + H * V) * 4;
  if (smem > 200 * 1024) return US_ERR_LIMIT;
  MixArgs a{q, kc, vc, talk, out, cu, pos, page_table, ldq, ldo, B, H, G, D, V, page, max_pages,
            size, keep, bf16, seq_lens, scale};
  static bool configured = false;
  if (!configured) {
    US_CUDA_CHECK(cudaFuncSetAttribute(head_mix_row_kernel,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    configured = true;
  }
  US_CUDA_CHECK(us::launch_pdl(head_mix_row_kernel, dim3(rows), dim3(kThreads), smem,
                               (cudaStream_t)stream_, a));
  return US_OK;
}
