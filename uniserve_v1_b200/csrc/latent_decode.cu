// Absorbed latent attention (see latent_attn.cu) for single query rows, bf16: every head of a row
// reads the same keys, so a key tile [64 tokens][latent | rotated part] is fetched once for up to
// 32 heads and serves as keys and, by its latent columns, as values.
//
// A CTA takes one split of a row's keys and 16 MT heads; the splits of a row are one thread-block
// cluster that merges its partial outputs in order.  Per tile: warps form scores for a slice of
// the channels each (the queries' fragments stay in registers), the softmax sums the slices per
// (head, key) in FP32, and every warp adds its columns of the value product.  The next tile is
// on its way (cp.async) meanwhile.
#include "include/us_common.cuh"
#include "include/us_mma.cuh"
#include "include/us_tc05.cuh"

namespace {

constexpr int kThreads = 512, kWarps = kThreads / 32;
constexpr int kTile = 64;            // keys
constexpr int kRot = 64;             // rotated channels, padded
constexpr int kPRow = kTile * 2 + 16;
constexpr int kSRow = kTile + 8;     // floats of a head's scores (rows apart hit other banks)
constexpr int kMostSplits = 16;      // more than 8 CTAs to a cluster where the device allows them

struct DecodeArgs {
  const __nv_bfloat16 *ql, *qr;
  long long ldql, ldqr;
  int hsql, hsqr;
  const __nv_bfloat16 *cp, *rp;
  int ldc, ldr;
  __nv_bfloat16* out;
  long long ldo;
  int hso;
  const int *rows, *cu, *pos, *seq_lens, *page_table;
  int B, H, R, RD, page, max_pages, window, splits;
  float scale_log2;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int RP, int MT>
__global__ void __launch_bounds__(kThreads, 1) latent_decode_kernel(const DecodeArgs a) {
  US_PDL_PROLOGUE();
  constexpr int PC = RP / 8 + kRot / 8;          // 16-byte pieces per key
  constexpr int NK = RP / 16 + kRot / 16;        // 16-channel steps of a score
  constexpr int KG = 8 / MT, NS = (NK + KG - 1) / KG;
  constexpr int NT = RP >= 128 ? RP / 128 : 1;   // 8-column value tiles per warp
  constexpr int HT = 16 * MT;
  constexpr uint32_t kKeyBytes = kTile * PC * 16;
  extern __shared__ __align__(1024) uint8_t sm[];
  const uint32_t sk = tc::smem_u32(sm);                         // 2 x key tile
  float* part = reinterpret_cast<float*>(sm + 2 * kKeyBytes);   // [KG][HT][kSRow] score slices
  const uint32_t sp = tc::smem_u32(part + KG * HT * kSRow);     // [HT][kPRow] weights, bf16
  float* mx = reinterpret_cast<float*>(sm + 2 * kKeyBytes + KG * HT * kSRow * 4 + HT * kPRow);
  float* sum = mx + HT;
  float* fac = sum + HT;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int lrow = lane & 15, lhalf = lane >> 4, r0 = lane >> 2, cq = (lane & 3) * 2;
  const int split = blockIdx.x, h0 = blockIdx.y * HT, nh = min(HT, a.H - h0);
  const long long t = blockIdx.z;         // row of ql, qr and out
  const int row = a.rows ? a.rows[t] : (int)t;                  // row of the packed batch
  int s = blockIdx.z;
  if (a.rows) {
    int lo = 0, hi = a.B - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (a.cu[mid] <= row) lo = mid; else hi = mid - 1;
    }
    s = lo;
  }
  const bool live = !a.seq_lens || a.seq_lens[s] > 0;           // the same in the whole cluster
  const int i = live ? a.pos[row] : -1;
  const int first = a.window > 0 ? max(0, i - a.window + 1) : 0;
  const int n = i + 1 - first;
  const int per = ((n + a.splits - 1) / a.splits + kTile - 1) / kTile * kTile;
  const int k0 = min(n, split * per), k1 = min(n, k0 + per);    // this split's keys, from `first`
  const int* pt = a.page_table + (long long)s * a.max_pages;

  // a thread copies eight pieces apart of one key of the tile
  const int krow = tid >> 3, kpc = tid & 7;
  // cache row of this thread's key of the tile at j0; looked up a tile ahead of its copies
  auto where = [&](int j0) -> long long {
    if (j0 + krow >= k1) return -1;
    const int key = first + j0 + krow, p = key / a.page;
    return (long long)pt[p] * a.page + (key - p * a.page);
  };
  auto fetch = [&](long long at, int buf) {
    const uint32_t dst = sk + buf * kKeyBytes;
    const bool in = at >= 0;
    const __nv_bfloat16 *c = a.cp + at * a.ldc, *r = a.rp + at * a.ldr;
#pragma unroll
    for (int x = 0; x < PC / 8; ++x) {
      const int pc = kpc + x * 8;
      const uint32_t d = dst + us::swz(krow, pc, PC);
      if (pc < RP / 8) {
        if (in && pc * 8 < a.ldc) us::cp16(d, c + pc * 8);
        else us::zero16(d);
      } else {
        if (in && (pc - RP / 8) * 8 < a.ldr) us::cp16(d, r + (pc - RP / 8) * 8);
        else us::zero16(d);
      }
    }
    us::cp_commit();
  };
  fetch(where(k0), 0);
  long long ahead = where(k0 + kTile);
  // queries: warp (m, g) keeps head tile m's fragments of channel steps g, g + KG, ... (two warps
  // each, for half of a tile's keys)
  const int wm = warp % MT, wg = (warp / MT) % KG, wk = (warp / 8) * 32;
  const bool has_values = warp * NT * 8 < RP;
  uint32_t qf[NS][4];
#pragma unroll
  for (int x = 0; x < NS; ++x) {
    const int st = wg + x * KG;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = wm * 16 + r0 + (e & 1) * 8, ch = st * 16 + cq + (e >> 1) * 8;
      uint32_t v = 0;
      if (live && st < NK && h < nh) {
        if (ch < RP) {
          if (ch < a.ldc)
            v = *reinterpret_cast<const uint32_t*>(a.ql + t * a.ldql + (long long)(h0 + h) * a.hsql + ch);
        } else if (ch - RP < a.ldr) {
          v = *reinterpret_cast<const uint32_t*>(a.qr + t * a.ldqr + (long long)(h0 + h) * a.hsqr + ch - RP);
        }
      }
      qf[x][e] = v;
    }
  }
  for (int h = tid; h < HT; h += kThreads) {
    mx[h] = -INFINITY;
    sum[h] = 0.f;
  }
  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int x = 0; x < NT; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[m][x][e] = 0.f;

  int buf = 0;
  for (int j0 = k0; j0 < k1; j0 += kTile, buf ^= 1) {
    us::cp_wait<0>();
    __syncthreads();                      // this tile is there; the other buffer and P are free
    if (j0 + kTile < k1) {
      fetch(ahead, buf ^ 1);
      ahead = where(j0 + 2 * kTile);
    }
    const uint32_t kb = sk + buf * kKeyBytes;
    {
      float sc[4][4];
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[x][e] = 0.f;
#pragma unroll
      for (int x = 0; x < NS; ++x) {
        const int st = wg + x * KG;
        if (st >= NK) break;
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          uint32_t b[4];
          us::ldsm4(b, kb + us::swz(wk + y * 16 + lrow, 2 * st + lhalf, PC));
          us::mma16816(sc[2 * y], qf[x][0], qf[x][1], qf[x][2], qf[x][3], b[0], b[2]);
          us::mma16816(sc[2 * y + 1], qf[x][0], qf[x][1], qf[x][2], qf[x][3], b[1], b[3]);
        }
      }
      float* p = part + (wg * HT + wm * 16 + r0) * kSRow + wk + cq;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        *reinterpret_cast<float2*>(p + x * 8) = make_float2(sc[x][0], sc[x][1]);
        *reinterpret_cast<float2*>(p + 8 * kSRow + x * 8) = make_float2(sc[x][2], sc[x][3]);
      }
    }
    __syncthreads();
    {                                     // lane: two keys, warp: every sixteenth head
      constexpr int HW = HT / kWarps;
      float v[HW][2], m[HW], m0[HW], l[HW];
#pragma unroll
      for (int x = 0; x < HW; ++x) {
        const int h = warp + x * kWarps;
        float2 q = make_float2(0.f, 0.f);
#pragma unroll
        for (int g = 0; g < KG; ++g) {
          const float2 e = *reinterpret_cast<const float2*>(part + (g * HT + h) * kSRow + lane * 2);
          q.x += e.x;
          q.y += e.y;
        }
        v[x][0] = j0 + lane * 2 < k1 ? q.x * a.scale_log2 : -INFINITY;
        v[x][1] = j0 + lane * 2 + 1 < k1 ? q.y * a.scale_log2 : -INFINITY;
        m[x] = fmaxf(v[x][0], v[x][1]);
        m0[x] = mx[h];
      }
#pragma unroll
      for (int o2 = 16; o2 > 0; o2 >>= 1)
#pragma unroll
        for (int x = 0; x < HW; ++x) m[x] = fmaxf(m[x], __shfl_xor_sync(0xffffffffu, m[x], o2));
#pragma unroll
      for (int x = 0; x < HW; ++x) {
        m[x] = fmaxf(m[x], m0[x]);
        v[x][0] = ex2(v[x][0] - m[x]);
        v[x][1] = ex2(v[x][1] - m[x]);
        l[x] = v[x][0] + v[x][1];
      }
#pragma unroll
      for (int o2 = 16; o2 > 0; o2 >>= 1)
#pragma unroll
        for (int x = 0; x < HW; ++x) l[x] += __shfl_xor_sync(0xffffffffu, l[x], o2);
#pragma unroll
      for (int x = 0; x < HW; ++x) {
        const int h = warp + x * kWarps;
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(sp + h * kPRow + lane * 4),
                     "r"(us::pack_bf(v[x][0], v[x][1])) : "memory");
        if (lane == 0) {
          const float f = ex2(m0[x] - m[x]);
          fac[h] = f;
          sum[h] = sum[h] * f + l[x];
          mx[h] = m[x];
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float f0 = fac[m * 16 + r0], f1 = fac[m * 16 + r0 + 8];
      if (!__any_sync(0xffffffffu, f0 != 1.f || f1 != 1.f)) continue;   // no maximum of the tile grew
#pragma unroll
      for (int x = 0; x < NT; ++x) {
        o[m][x][0] *= f0;
        o[m][x][1] *= f0;
        o[m][x][2] *= f1;
        o[m][x][3] *= f1;
      }
    }
    if (!has_values) continue;
    uint32_t p[MT][4][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int k = 0; k < 4; ++k) us::ldsm4(p[m][k], sp + (m * 16 + lrow) * kPRow + (k * 16 + lhalf * 8) * 2);
#pragma unroll
    for (int x = 0; x < NT; ++x)
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        uint32_t b[4];                    // 32 keys x 8 columns
        us::ldsm4t(b, kb + us::swz(y * 32 + lane, warp * NT + x, PC));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          us::mma16816(o[m][x], p[m][2 * y][0], p[m][2 * y][1], p[m][2 * y][2], p[m][2 * y][3], b[0], b[1]);
          us::mma16816(o[m][x], p[m][2 * y + 1][0], p[m][2 * y + 1][1], p[m][2 * y + 1][2],
                       p[m][2 * y + 1][3], b[2], b[3]);
        }
      }
  }
  __syncthreads();                        // the key tiles become the partial outputs
  float* os = reinterpret_cast<float*>(sm);                      // [HT][RP]
  if (has_values) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int x = 0; x < NT; ++x)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          *reinterpret_cast<float2*>(os + (m * 16 + r0 + e * 8) * RP + (warp * NT + x) * 8 + cq) =
              make_float2(o[m][x][e * 2], o[m][x][e * 2 + 1]);
  }
  __syncthreads();
  if (a.splits > 1) tc::cluster_sync();
  // every CTA of the cluster finishes a share of the heads' columns, adding the splits in order: first the
  // splits' maxima and sums side by side (in `part`), then each split's factor per head, then the columns
  float* mt = part;                                              // [HT][kMostSplits] each
  float* lt = mt + HT * kMostSplits;
  float* wgt = lt + HT * kMostSplits;
  for (int e = tid; e < nh * a.splits; e += kThreads) {
    const int h = e / a.splits, p = e - h * a.splits;
    const uint32_t am = (uint32_t)__cvta_generic_to_shared(&mx[h]);
    const uint32_t al = (uint32_t)__cvta_generic_to_shared(&sum[h]);
    mt[h * kMostSplits + p] = a.splits > 1 ? tc::ld_dsmem_f32(tc::map_to_cta(am, p)) : mx[h];
    lt[h * kMostSplits + p] = a.splits > 1 ? tc::ld_dsmem_f32(tc::map_to_cta(al, p)) : sum[h];
  }
  __syncthreads();
  for (int h = tid; h < nh; h += kThreads) {
    const float *m = mt + h * kMostSplits, *l = lt + h * kMostSplits;
    float top = -INFINITY, den = 0.f;
    for (int p = 0; p < a.splits; ++p) top = fmaxf(top, m[p]);
    if (top > -INFINITY)
      for (int p = 0; p < a.splits; ++p) den = fmaf(ex2(m[p] - top), l[p], den);
    for (int p = 0; p < a.splits; ++p) wgt[h * kMostSplits + p] = den > 0.f ? ex2(m[p] - top) / den : 0.f;
  }
  __syncthreads();
  const int cols = a.hso, quads = (cols + 3) / 4;
  const bool wide = ((a.ldo | cols) & 3) == 0;
  for (int e = tid + split * kThreads; e < nh * quads; e += kThreads * a.splits) {
    const int h = e / quads, c = (e - h * quads) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < RP) {
      const uint32_t ao = (uint32_t)__cvta_generic_to_shared(os + h * RP + c);
      auto add = [&](int p0) {                       // eight splits, fetched together
        float4 o4[8];
#pragma unroll
        for (int p = 0; p < 8; ++p)
          if (p0 + p < a.splits)
            o4[p] = a.splits > 1 ? tc::ld_dsmem_f32x4(tc::map_to_cta(ao, p0 + p))
                                 : *reinterpret_cast<const float4*>(os + h * RP + c);
#pragma unroll
        for (int p = 0; p < 8; ++p)
          if (p0 + p < a.splits) {
            const float f = wgt[h * kMostSplits + p0 + p];
            v.x = fmaf(f, o4[p].x, v.x);
            v.y = fmaf(f, o4[p].y, v.y);
            v.z = fmaf(f, o4[p].z, v.z);
            v.w = fmaf(f, o4[p].w, v.w);
          }
      };
      add(0);
      if (a.splits > 8) add(8);
    }
    __nv_bfloat16* dst = a.out + t * a.ldo + (long long)(h0 + h) * a.hso + c;
    const float f[4] = {c < a.R ? v.x : 0.f, c + 1 < a.R ? v.y : 0.f, c + 2 < a.R ? v.z : 0.f,
                        c + 3 < a.R ? v.w : 0.f};
    if (wide) {
      *reinterpret_cast<uint2*>(dst) = make_uint2(us::pack_bf(f[0], f[1]), us::pack_bf(f[2], f[3]));
    } else {
#pragma unroll
      for (int q = 0; q < 4; ++q)
        if (c + q < cols) dst[q] = us::f2bf(f[q]);
    }
  }
  if (a.splits > 1) tc::cluster_sync();   // nobody leaves while its sums may still be read
}

template <int RP, int MT>
int launch_decode(DecodeArgs a, int rows, cudaStream_t stream) {
  constexpr int PC = RP / 8 + kRot / 8, HT = 16 * MT;
  constexpr size_t smem = 2 * (size_t)kTile * PC * 16 + (8 / MT) * HT * kSRow * 4 + HT * kPRow + 3 * HT * 4;
  static_assert(2 * kTile * PC * 16 >= HT * RP * 4, "partial outputs fit the key tiles");
  static bool configured = false;
  if (!configured) {
    US_CUDA_CHECK(cudaFuncSetAttribute(latent_decode_kernel<RP, MT>,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = true;
  }
  if (a.splits > 8) {
    static const int most = us::cluster_limit(latent_decode_kernel<RP, MT>, kMostSplits, kThreads, smem);
    if (a.splits > most) a.splits = most;
  }
  static_assert((8 / MT) * kSRow >= 3 * kMostSplits, "the splits' factors fit the score slices");
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(a.splits, us::ceil_div(a.H, HT), rows);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = us::pdl_enabled() ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = a.splits;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = a.splits > 1 ? 2 : 1;
  US_CUDA_CHECK(cudaLaunchKernelEx(&cfg, latent_decode_kernel<RP, MT>, a));
  return US_OK;
}

}  // namespace

// `count` single rows: rows `rows` of the packed batch (sequence s has cu[s] .. cu[s + 1]), packed in ql, qr
// and out; rows null: row i is sequence i's only one.
US_API int us_latent_decode(const void* ql, long long ldql, int hsql, const void* qr, long long ldqr,
                            int hsqr, const void* cpages, int ldc, const void* rpages, int ldr,
                            void* out, long long ldo, int hso, const int* rows, const int* cu,
                            const int* pos, const int* seq_lens, const int* page_table, int count,
                            int B, int H, int R, int RD, int page, int max_pages, int window,
                            int splits, float scale, void* stream_) {
  US_REQUIRE(ql && qr && cpages && rpages && out && cu && pos && page_table && count >= 0 && B >= 1 &&
             H >= 1 && R >= 1 && RD >= 0 && page >= 1 && hso >= R && ldc >= R && ldr >= RD &&
             ((uintptr_t)out % 8) == 0 && splits >= 1 && splits <= kMostSplits && count <= 65535 && (rows || count == B));
  US_REQUIRE((ldc % 8) == 0 && (ldr % 8) == 0 && (ldql % 2) == 0 && (hsql % 2) == 0 && (ldqr % 2) == 0 &&
             (hsqr % 2) == 0 && ((uintptr_t)cpages % 16) == 0 && ((uintptr_t)rpages % 16) == 0 &&
             ((uintptr_t)ql % 4) == 0 && ((uintptr_t)qr % 4) == 0);
  if (ldc > 512 || ldr > kRot) return US_ERR_LIMIT;
  if (count == 0) return US_OK;
  DecodeArgs a{(const __nv_bfloat16*)ql, (const __nv_bfloat16*)qr, ldql, ldqr, hsql, hsqr,
               (const __nv_bfloat16*)cpages, (const __nv_bfloat16*)rpages, ldc, ldr,
               (__nv_bfloat16*)out, ldo, hso, rows, cu, pos, seq_lens, page_table, B, H, R, RD, page,
               max_pages, window, splits, scale * 1.4426950408889634f};
  cudaStream_t stream = (cudaStream_t)stream_;
  // 16 heads to a CTA while there are few (clusters of one CTA per SM do not fill every SM of a GPC)
  const bool narrow = H <= 16 || (long long)count * us::ceil_div(H, 16) * splits <= 64;
#define US_LATENT(RP) return narrow ? launch_decode<RP, 1>(a, count, stream) : launch_decode<RP, 2>(a, count, stream)
  if (ldc <= 64) US_LATENT(64);
  if (ldc <= 128) US_LATENT(128);
  if (ldc <= 256) US_LATENT(256);
  US_LATENT(512);
#undef US_LATENT
}
