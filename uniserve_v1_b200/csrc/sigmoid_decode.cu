// Attention of single query rows over cache pages with weights that do not depend on the other keys, bf16:
//
//   w_h(i, j) = sigmoid(cap tanh(scale temp_h (q_h(i) . k_g(j)) / cap) + shift_h),   j <= i
//   o_h(i)    = sigmoid(gate_h(i)) sum_j w_h(i, j) v_g(j),   g = h / (H / G)
//
// Without a softmax nothing ties the keys together: every warp takes tiles of 16 keys of its own through a
// ring of asynchronous copies, forms scores, weights and its share of the value product in registers (the
// score fragments are the value product's operand as they stand), and no warp waits for another before
// the end.  A CTA serves one row's heads of one key head (16 at a time) over one split of the keys; warps
// add up in shared memory, the splits are a cluster that adds up in order.
#include "include/us_common.cuh"
#include "include/us_mma.cuh"
#include "include/us_tc05.cuh"

namespace {

constexpr int kWarps = 4, kThreads = kWarps * 32;
constexpr int kKeys = 16;            // per tile
constexpr int kStages = 3;           // tiles in a warp's ring
constexpr int kHeads = 16;
constexpr int kMostSplits = 16;      // more than 8 CTAs to a cluster where the device allows them

struct SigDecode {
  const __nv_bfloat16* q;            // [T, H, ..]: rows at ldq, heads at hsq
  long long ldq;
  int hsq;
  const __nv_bfloat16 *kp, *vp;      // pages [n, page, G, D], [n, page, G, V]
  __nv_bfloat16* out;                // [T, ldo], head h at column h V
  long long ldo;
  const int *rows, *cu, *pos, *seq_lens, *page_table;
  int B, H, G, D, V, page, max_pages, window, splits;
  const float *temp, *shift;
  float scale, cap, out_scale;
  const __nv_bfloat16* gate;         // [rows of the batch, H] at ldg, or null
  long long ldg;
};

template <int DP, int VP>
__global__ void __launch_bounds__(kThreads) sigmoid_decode_kernel(const SigDecode a) {
  US_PDL_PROLOGUE();
  constexpr int KP = DP / 8, PV = VP / 8;              // 16-byte pieces of a key's and a value's row
  constexpr uint32_t kStage = kKeys * (KP + PV) * 16;
  extern __shared__ __align__(1024) uint8_t sm[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int lrow = lane & 15, lhalf = lane >> 4, r0 = lane >> 2, cq = (lane & 3) * 2;
  const int rep = a.H / a.G, parts = (rep + kHeads - 1) / kHeads;
  const int g = blockIdx.y / parts, part = blockIdx.y - g * parts;
  const int h0 = g * rep + part * kHeads, nh = min(kHeads, rep - part * kHeads);
  const int split = blockIdx.x;
  const long long t = blockIdx.z;                      // row of q and out
  const int row = a.rows ? a.rows[t] : (int)t;         // row of the packed batch
  int s = blockIdx.z;
  if (a.rows) {
    int lo = 0, hi = a.B - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (a.cu[mid] <= row) lo = mid; else hi = mid - 1;
    }
    s = lo;
  }
  const bool live = !a.seq_lens || a.seq_lens[s] > 0;
  const int i = live ? a.pos[row] : -1;
  const int first = a.window > 0 ? max(0, i - a.window + 1) : 0;
  const int n = i + 1 - first;
  const int per = ((n + a.splits - 1) / a.splits + kKeys - 1) / kKeys * kKeys;
  const int k0 = min(n, split * per), k1 = min(n, k0 + per);       // this split's keys, from `first`
  const int* pt = a.page_table + (long long)s * a.max_pages;
  const uint32_t ring = tc::smem_u32(sm) + warp * kStages * kStage;

  // lane l < 16 knows the cache row of the tile's key l, looked up a tile ahead of its copies
  auto where = [&](int j0) -> int {
    const int key = first + j0 + lrow;
    if (j0 + lrow >= k1) return -1;
    const int p = key / a.page;
    return pt[p] * a.page + (key - p * a.page);
  };
  auto fetch = [&](int at, int stage) {
    const uint32_t sk = ring + stage * kStage, sv = sk + kKeys * KP * 16;
#pragma unroll
    for (int x = 0; x < kKeys * KP / 32; ++x) {
      const int e = x * 32 + lane, r = e / KP, c = e - r * KP;
      const long long src = __shfl_sync(0xffffffffu, at, r);
      const uint32_t d = sk + us::swz(r, c, KP);
      if (src >= 0 && c * 8 < a.D) us::cp16(d, a.kp + (src * a.G + g) * a.D + c * 8);
      else us::zero16(d);
    }
#pragma unroll
    for (int x = 0; x < kKeys * PV / 32; ++x) {
      const int e = x * 32 + lane, r = e / PV, c = e - r * PV;
      const long long src = __shfl_sync(0xffffffffu, at, r);
      const uint32_t d = sv + us::swz(r, c, PV);
      if (src >= 0 && c * 8 < a.V) us::cp16(d, a.vp + (src * a.G + g) * a.V + c * 8);
      else us::zero16(d);
    }
  };
  const int step = kWarps * kKeys, j_first = k0 + warp * kKeys;
  int ahead = where(j_first);
#pragma unroll
  for (int x = 0; x < kStages - 1; ++x) {
    const int at = ahead;
    ahead = where(j_first + (x + 1) * step);
    if (j_first + x * step < k1) fetch(at, x);
    us::cp_commit();
  }
  // queries as operand fragments: rows are heads
  uint32_t qf[DP / 16][4];
#pragma unroll
  for (int st = 0; st < DP / 16; ++st)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = r0 + (e & 1) * 8, ch = st * 16 + cq + (e >> 1) * 8;
      qf[st][e] = live && h < nh && ch < a.D
                      ? *reinterpret_cast<const uint32_t*>(a.q + t * a.ldq + (long long)(h0 + h) * a.hsq + ch) : 0u;
    }
  float fac[2], shift[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int h = r0 + e * 8;
    fac[e] = h < nh ? a.scale * a.temp[h0 + h] : 0.f;
    if (a.cap > 0.f) fac[e] /= a.cap;
    shift[e] = h < nh ? a.shift[h0 + h] : 0.f;
  }
  float o[VP / 8][4];
#pragma unroll
  for (int x = 0; x < VP / 8; ++x)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[x][e] = 0.f;

  int stage = 0;
  for (int j0 = j_first; j0 < k1; j0 += step) {
    us::cp_wait<kStages - 2>();
    __syncwarp();                        // the tile is there for all lanes; the stage before it is free
    {
      const int j2 = j0 + (kStages - 1) * step, at = ahead;
      ahead = where(j2 + step);
      if (j2 < k1) fetch(at, stage == 0 ? kStages - 1 : stage - 1);
      us::cp_commit();
    }
    const uint32_t sk = ring + stage * kStage, sv = sk + kKeys * KP * 16;
    float sc[2][4] = {};
#pragma unroll
    for (int st = 0; st < DP / 16; ++st) {
      uint32_t b[4];
      us::ldsm4(b, sk + us::swz(lrow, 2 * st + lhalf, KP));
      us::mma16816(sc[0], qf[st][0], qf[st][1], qf[st][2], qf[st][3], b[0], b[2]);
      us::mma16816(sc[1], qf[st][0], qf[st][1], qf[st][2], qf[st][3], b[1], b[3]);
    }
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float z = sc[x][e] * fac[e >> 1];
        if (a.cap > 0.f) z = a.cap * tanhf(z);
        const bool in = j0 + x * 8 + cq + (e & 1) < k1;
        sc[x][e] = in ? 1.f / (1.f + __expf(-(z + shift[e >> 1]))) : 0.f;
      }
    const uint32_t p0 = us::pack_bf(sc[0][0], sc[0][1]), p1 = us::pack_bf(sc[0][2], sc[0][3]);
    const uint32_t p2 = us::pack_bf(sc[1][0], sc[1][1]), p3 = us::pack_bf(sc[1][2], sc[1][3]);
#pragma unroll
    for (int x = 0; x < VP / 16; ++x) {
      uint32_t b[4];
      us::ldsm4t(b, sv + us::swz(lrow, 2 * x + lhalf, PV));
      us::mma16816(o[2 * x], p0, p1, p2, p3, b[0], b[1]);
      us::mma16816(o[2 * x + 1], p0, p1, p2, p3, b[2], b[3]);
    }
    stage = stage + 1 == kStages ? 0 : stage + 1;
  }
  us::cp_wait<0>();
  __syncthreads();                       // the rings become the partial outputs
  float* os = reinterpret_cast<float*>(sm);            // [kWarps][kHeads][VP]
#pragma unroll
  for (int x = 0; x < VP / 8; ++x)
#pragma unroll
    for (int e = 0; e < 2; ++e)
      *reinterpret_cast<float2*>(os + ((warp * kHeads) + r0 + e * 8) * VP + x * 8 + cq) =
          make_float2(o[x][e * 2], o[x][e * 2 + 1]);
  __syncthreads();
  for (int e = tid * 4; e < kHeads * VP; e += kThreads * 4) {
    float4 v = *reinterpret_cast<const float4*>(os + e);
#pragma unroll
    for (int w = 1; w < kWarps; ++w) {
      const float4 u = *reinterpret_cast<const float4*>(os + w * kHeads * VP + e);
      v = make_float4(v.x + u.x, v.y + u.y, v.z + u.z, v.w + u.w);
    }
    *reinterpret_cast<float4*>(os + e) = v;
  }
  if (a.splits > 1) tc::cluster_sync();
  else __syncthreads();
  // every CTA of the cluster finishes a share of the columns
  const int quads = (a.V + 3) / 4;
  const bool wide = ((a.ldo | a.V) & 3) == 0 && ((uintptr_t)a.out & 7) == 0;
  for (int e = tid + split * kThreads; e < nh * quads; e += kThreads * a.splits) {
    const int h = e / quads, c = (e - h * quads) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (a.splits == 1) {
      v = *reinterpret_cast<const float4*>(os + h * VP + c);
    } else {
      const uint32_t at = (uint32_t)__cvta_generic_to_shared(os + h * VP + c);
      for (int p = 0; p < a.splits; ++p) {
        const float4 u = tc::ld_dsmem_f32x4(tc::map_to_cta(at, (uint32_t)p));
        v = make_float4(v.x + u.x, v.y + u.y, v.z + u.z, v.w + u.w);
      }
    }
    float f = a.out_scale;
    if (a.gate) f /= 1.f + __expf(-us::bf2f(a.gate[(long long)row * a.ldg + h0 + h]));
    __nv_bfloat16* dst = a.out + t * a.ldo + (long long)(h0 + h) * a.V + c;
    if (wide) {
      *reinterpret_cast<uint2*>(dst) = make_uint2(us::pack_bf(v.x * f, v.y * f), us::pack_bf(v.z * f, v.w * f));
    } else {
      const float w[4] = {v.x * f, v.y * f, v.z * f, v.w * f};
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (c + k < a.V) dst[k] = us::f2bf(w[k]);
    }
  }
  if (a.splits > 1) tc::cluster_sync();  // nobody leaves while its sums may still be read
}

template <int DP, int VP>
int launch(SigDecode a, int rows, cudaStream_t stream) {
  constexpr size_t smem = (size_t)kWarps * kStages * kKeys * (DP + VP) * 2;
  static_assert(smem >= (size_t)kWarps * kHeads * VP * 4, "partial outputs fit the rings");
  static bool configured = false;
  if (!configured) {
    US_CUDA_CHECK(cudaFuncSetAttribute(sigmoid_decode_kernel<DP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                       (int)smem));
    configured = true;
  }
  if (a.splits > 8) {
    static const int most = us::cluster_limit(sigmoid_decode_kernel<DP, VP>, kMostSplits, kThreads, smem);
    if (a.splits > most) a.splits = most;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(a.splits, a.G * us::ceil_div(a.H / a.G, kHeads), rows);
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
  US_CUDA_CHECK(cudaLaunchKernelEx(&cfg, sigmoid_decode_kernel<DP, VP>, a));
  return US_OK;
}

}  // namespace

// `count` single rows: rows `rows` of the packed batch (sequence s has cu[s] .. cu[s + 1]), packed in q and out;
// rows null: row i is sequence i's only one.  D and V multiples of 8 up to 128.  seq_lens [B] or null: length 0
// marks padding, whose rows become zero.  cap 0: scores as they are.  gate: of the packed batch's rows, or null.
US_API int us_sigmoid_decode(const void* q, long long ldq, int hsq, const void* kpages, const void* vpages,
                             void* out, long long ldo, const int* rows, const int* cu, const int* pos,
                             const int* seq_lens, const int* page_table, int count, int B, int H, int G,
                             int D, int V, int page, int max_pages, int window, int splits, float scale,
                             const float* temp, const float* shift, float cap, float out_scale,
                             const void* gate, long long ldg, void* stream_) {
  US_REQUIRE(q && kpages && vpages && out && cu && pos && page_table && temp && shift && count >= 0 && B >= 1 &&
             H >= 1 && G >= 1 && H % G == 0 && D >= 8 && V >= 8 && page >= 1 && splits >= 1 && splits <= kMostSplits &&
             count <= 65535 && G * us::ceil_div(H / G, kHeads) <= 65535 && (rows || count == B) &&
             ldo >= (long long)H * V && cap >= 0.f);
  US_REQUIRE((D % 8) == 0 && (V % 8) == 0 && (ldq % 2) == 0 && (hsq % 2) == 0 && ((uintptr_t)q % 4) == 0 &&
             ((uintptr_t)kpages % 16) == 0 && ((uintptr_t)vpages % 16) == 0);
  if (D > 128 || V > 128) return US_ERR_LIMIT;
  if (count == 0) return US_OK;
  SigDecode a{(const __nv_bfloat16*)q, ldq, hsq, (const __nv_bfloat16*)kpages, (const __nv_bfloat16*)vpages,
              (__nv_bfloat16*)out, ldo, rows, cu, pos, seq_lens, page_table, B, H, G, D, V, page, max_pages, window,
              splits, temp, shift, scale, cap, out_scale, (const __nv_bfloat16*)gate, ldg};
  cudaStream_t stream = (cudaStream_t)stream_;
  if (D <= 64) return V <= 64 ? launch<64, 64>(a, count, stream) : launch<64, 128>(a, count, stream);
  return V <= 64 ? launch<128, 64>(a, count, stream) : launch<128, 128>(a, count, stream);
}
