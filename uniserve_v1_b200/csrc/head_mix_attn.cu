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
// Keys are read through the page table; the key list of a query is its kept keys followed by its
// window.  Three forms:
//
// * row form (any head width, bf16 or FP32 pages): one CTA per query row, all heads, FP32 FMAs;
// * decode form (bf16, one row per sequence): CTAs per (key split, kv head, sequence) write the
//   scores and their statistics, then CTAs of the same shape turn every head's scores of their
//   keys into mixed weights (FP32) and form the value product; the splits of a sequence are one
//   thread-block cluster that sums its partial outputs in a fixed order.  Keys and values cross
//   HBM once;
// * tile form (bf16 prompts): a CTA takes 16 consecutive query rows and all heads.  A first sweep
//   over the keys finds the statistics, a second one forms the probabilities, mixes them and
//   multiplies the values, 16 keys at a time, on warp-level tensor instructions (every product
//   of this operator is 16 rows high: an output head's weights exist only after all heads' scores
//   of the same 16 x 16 tile do).  Probabilities and mixed weights enter the products as the sum
//   of two bf16 values, which keeps 16 bits of their fraction; T is a bf16 tensor and exact.
#include "include/us_common.cuh"
#include "include/us_tc05.cuh"

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

// ------------------------------------------------------------------ decode --
__device__ __forceinline__ void mma16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2,
                                         uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
      "{%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ uint32_t pack_bf(float a, float b) {
  __nv_bfloat162 p = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&p);
}
// x = hi + lo with both halves bf16
__device__ __forceinline__ void split_bf(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf(x - us::bf2f(h.x), y - us::bf2f(h.y));
}

// byte offset of 16-byte piece c of row r in a tile whose rows hold `pieces` pieces (8 or 16):
// pieces are XOR-swizzled by row so that 8 consecutive rows read 8 different bank groups
template <int PIECES>
__device__ __forceinline__ uint32_t swz(int r, int c) {
  return (uint32_t)(r * PIECES + (c ^ (r & 7))) * 16u;
}

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct StepArgs {
  const __nv_bfloat16* q;
  const __nv_bfloat16 *kc, *vc;
  const float* talk;
  __nv_bfloat16* out;
  float* scores;              // [B, H, cap]
  float* stats;               // [B, H, splits, 2]: maximum, sum of exponentials
  const int *pos, *page_table, *seq_lens;
  long long ldq, ldo;
  int B, H, G, D, V, page, max_pages, size, keep, cap, splits;
  float scale;
};

struct KeyList {
  int n, lo, kept;
  __device__ __forceinline__ int key(int x) const { return x < kept ? x : lo + x - kept; }
};
__device__ __forceinline__ KeyList key_list(int pos, int size, int keep, int cap) {
  KeyList k;
  k.lo = size > 0 ? max(0, pos - size + 1) : 0;
  k.kept = min(max(keep, 0), k.lo);
  k.n = min(cap, k.kept + pos - k.lo + 1);
  return k;
}

constexpr int kStepThreads = 128;
constexpr int kStepTile = 32;         // keys per step of the value product
// keys of one split: whole tiles
__host__ __device__ __forceinline__ int split_keys(int n, int splits) {
  return ((n + splits - 1) / splits + kStepTile - 1) / kStepTile * kStepTile;
}

// Scores of one split's keys for the heads of one kv head.  A warp takes 8 keys per product: a
// lane's 16-byte piece of a key row feeds two instructions, the queries' rows (at most 16 heads)
// sit in registers in the same order of channels.  kD8 = 16-byte pieces per lane.
template <int kD8>
__global__ void __launch_bounds__(kStepThreads) head_mix_scores_kernel(const StepArgs a) {
  US_PDL_PROLOGUE();
  extern __shared__ __align__(16) float sc[];            // [rep][keys of the split]
  const int split = blockIdx.x, u = blockIdx.y, b = blockIdx.z;
  if (a.seq_lens[b] <= 0) return;
  const int rep = a.H / a.G;
  const KeyList kl = key_list(a.pos[b], a.size, a.keep, a.cap);
  const int per = split_keys(kl.n, a.splits);
  const int k0 = min(kl.n, split * per), nk = min(kl.n, k0 + per) - k0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = lane >> 2, kq = lane & 3;
  uint4 qa[kD8], qb[kD8];
  const __nv_bfloat16* qr = a.q + (long long)b * a.ldq + (long long)u * rep * a.D;
#pragma unroll
  for (int i = 0; i < kD8; ++i) {
    const int d = (i * 4 + kq) * 8;
    const uint4 z = make_uint4(0, 0, 0, 0);
    qa[i] = (d < a.D && row < rep) ? *reinterpret_cast<const uint4*>(qr + (long long)row * a.D + d) : z;
    qb[i] = (d < a.D && row + 8 < rep) ? *reinterpret_cast<const uint4*>(qr + (long long)(row + 8) * a.D + d) : z;
  }
  const int* pt = a.page_table + (long long)b * a.max_pages;
  float* srow = a.scores + ((long long)b * a.H + (long long)u * rep) * a.cap;
  auto fetch = [&](int j0, uint4 (&kv)[kD8]) {
    const int key = kl.key(min(k0 + j0 + row, kl.n - 1));
    const __nv_bfloat16* kr =
        a.kc + (((long long)pt[key / a.page] * a.page + key % a.page) * a.G + u) * a.D;
#pragma unroll
    for (int i = 0; i < kD8; ++i) {
      const int d = (i * 4 + kq) * 8;
      kv[i] = d < a.D ? *reinterpret_cast<const uint4*>(kr + d) : make_uint4(0, 0, 0, 0);
    }
  };
  constexpr int kStride = kStepThreads / 4;      // 4 warps x 8 keys
  uint4 ahead[kD8];
  if (warp * 8 < nk) fetch(warp * 8, ahead);
  for (int j0 = warp * 8; j0 < nk; j0 += kStride) {
    uint4 kv[kD8];
#pragma unroll
    for (int i = 0; i < kD8; ++i) kv[i] = ahead[i];
    if (j0 + kStride < nk) fetch(j0 + kStride, ahead);
    float c[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < kD8; ++i) {
      mma16816(c, qa[i].x, qb[i].x, qa[i].y, qb[i].y, kv[i].x, kv[i].y);
      mma16816(c, qa[i].z, qb[i].z, qa[i].w, qb[i].w, kv[i].z, kv[i].w);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = row + (e >> 1) * 8, j = j0 + kq * 2 + (e & 1);
      if (h < rep && j < nk) {
        const float v = c[e] * a.scale;
        sc[h * per + j] = v;
        srow[(long long)h * a.cap + k0 + j] = v;
      }
    }
  }
  __syncthreads();
  for (int h = warp; h < rep; h += kStepThreads / 32) {
    float m = -INFINITY, l = 0.f;
    for (int j = lane; j < nk; j += 32) m = fmaxf(m, sc[h * per + j]);
    m = us::warp_max(m);
    for (int j = lane; j < nk; j += 32) l += expf(sc[h * per + j] - m);
    l = us::warp_sum(l);
    if (lane == 0) {
      float* st = a.stats + (((long long)b * a.H + u * rep + h) * a.splits + split) * 2;
      st[0] = m;
      st[1] = l;
    }
  }
}

constexpr int kWRow = kStepTile * 2 + 16;    // bytes of a head's 32 weights (bf16, padded)

// Mixed weights and value product of one split's keys for the heads of one kv head, 32 keys a
// step on warp-level tensor instructions.  Probabilities P [H][32] and mixed weights W [16][32]
// are the sum of two bf16 values.  For the mixture a warp takes 8 keys, for the value product a
// quarter of the value columns.  The next step's values (cp.async) and scores (registers) are on
// their way while a step computes.  NK: 16-head steps of the mixture, VP: value width padded.
template <int NK, int VP>
__global__ void __launch_bounds__(kStepThreads) head_mix_apply_kernel(const StepArgs a) {
  US_PDL_PROLOGUE();
  constexpr int VC = VP / 8, HK = NK * 16, NP = HK / 8, NT = VP / 32;
  extern __shared__ __align__(1024) uint8_t dsm[];
  const int split = blockIdx.x, u = blockIdx.y, b = blockIdx.z;
  const int rep = a.H / a.G, H = a.H;
  const uint32_t sv = tc::smem_u32(dsm);                     // 2 x [32 keys][VC pieces]
  constexpr uint32_t kVBytes = kStepTile * VP * 2;
  const uint32_t sp = sv + 2 * kVBytes;                      // [2: hi, lo][HK][kWRow]
  constexpr uint32_t kPHalf = HK * kWRow;
  const uint32_t sw = sp + 2 * kPHalf;                       // [2][16][kWRow]
  constexpr uint32_t kWHalf = 16 * kWRow;
  float* os = reinterpret_cast<float*>(dsm + 2 * kVBytes + 2 * kPHalf + 2 * kWHalf);   // [rep][V]
  __shared__ float mx[HK], inv[HK];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int lrow = lane & 15, lhalf = lane >> 4, r0 = lane >> 2, cq = (lane & 3) * 2;
  const bool live = a.seq_lens[b] > 0;         // the same in the whole cluster
  float o[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
  if (live) {
    const KeyList kl = key_list(a.pos[b], a.size, a.keep, a.cap);
    const int per = split_keys(kl.n, a.splits);
    const int k0 = min(kl.n, split * per), k1 = min(kl.n, k0 + per);
    const int* pt = a.page_table + (long long)b * a.max_pages;
    const float* srow = a.scores + (long long)b * H * a.cap;
    const int kp = (tid & 15) * 2, pg = tid >> 4;            // this thread's key pair, first head
    float2 ahead[NP];
    auto fetch_scores = [&](int j0) {
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int g = pg + i * 8;
        ahead[i] = (g < H && j0 + kp < k1)
                       ? *reinterpret_cast<const float2*>(srow + (long long)g * a.cap + j0 + kp)
                       : make_float2(-INFINITY, -INFINITY);
      }
    };
    auto fetch_values = [&](int j0, int buf) {
      constexpr int kRows = kStepThreads / VC;
      const int c = tid & (VC - 1);
#pragma unroll
      for (int i = 0; i < kStepTile / kRows; ++i) {
        const int r = tid / VC + i * kRows;
        const uint32_t dst = sv + buf * kVBytes + swz<VC>(r, c);
        if (j0 + r < k1 && c * 8 < a.V) {
          const int key = kl.key(j0 + r), p = key / a.page;
          cp16(dst, a.vc + (((long long)pt[p] * a.page + (key - p * a.page)) * a.G + u) * a.V + c * 8);
        } else {
          asm volatile("st.shared.v4.u32 [%0], {%1,%1,%1,%1};" ::"r"(dst), "r"(0) : "memory");
        }
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (k0 < k1) {
      fetch_values(k0, 0);
      fetch_scores(k0);
    }
    for (int g = tid; g < HK; g += kStepThreads) {
      float m = -INFINITY, l = 0.f;
      if (g < H) {
        const float2* st = reinterpret_cast<const float2*>(a.stats) + ((long long)b * H + g) * a.splits;
        float2 v[8];
#pragma unroll
        for (int s = 0; s < 8; ++s) v[s] = s < a.splits ? st[s] : make_float2(-INFINITY, 0.f);
#pragma unroll
        for (int s = 0; s < 8; ++s) m = fmaxf(m, v[s].x);
#pragma unroll
        for (int s = 0; s < 8; ++s)
          if (v[s].y > 0.f) l += v[s].y * expf(v[s].x - m);
      }
      mx[g] = g < H ? m : 0.f;
      inv[g] = g < H ? 1.f / l : 0.f;
    }
    uint32_t tf[NK][4];                                       // T[u * rep + 0..15][g]
#pragma unroll
    for (int k = 0; k < NK; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int h = r0 + (e & 1) * 8, g = k * 16 + cq + (e >> 1) * 8;
        const float* t = a.talk + (long long)(u * rep + h) * H + g;
        tf[k][e] = pack_bf(h < rep && g < H ? t[0] : 0.f, h < rep && g + 1 < H ? t[1] : 0.f);
      }
    __syncthreads();
    float mg[NP], ig[NP];
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      mg[i] = mx[pg + i * 8];
      ig[i] = inv[pg + i * 8];
    }
    int buf = 0;
    for (int j0 = k0; j0 < k1; j0 += kStepTile, buf ^= 1) {
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const float x = expf(ahead[i].x - mg[i]) * ig[i];
        const float y = j0 + kp + 1 < k1 ? expf(ahead[i].y - mg[i]) * ig[i] : 0.f;
        uint32_t hi, low;
        split_bf(x, y, hi, low);
        const uint32_t dst = sp + (pg + i * 8) * kWRow + kp * 2;
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(dst), "r"(hi) : "memory");
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(dst + kPHalf), "r"(low) : "memory");
      }
      asm volatile("cp.async.wait_group 0;" ::: "memory");
      __syncthreads();                         // P and this step's values; the other buffer is free
      if (j0 + kStepTile < k1) {
        fetch_values(j0 + kStepTile, buf ^ 1);
        fetch_scores(j0 + kStepTile);
      }
      float w[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        uint32_t bp[4];                        // hi (first two) and lo of 16 heads x the warp's 8 keys
        ldsm4t(bp, sp + lhalf * kPHalf + (k * 16 + lrow) * kWRow + warp * 16);
        mma16816(w, tf[k][0], tf[k][1], tf[k][2], tf[k][3], bp[0], bp[1]);
        mma16816(w, tf[k][0], tf[k][1], tf[k][2], tf[k][3], bp[2], bp[3]);
      }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        uint32_t hi, low;
        split_bf(w[r * 2], w[r * 2 + 1], hi, low);
        const uint32_t dst = sw + (r0 + r * 8) * kWRow + (warp * 8 + cq) * 2;
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(dst), "r"(hi) : "memory");
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(dst + kWHalf), "r"(low) : "memory");
      }
      __syncthreads();
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        uint32_t wh[4], wl[4];
        ldsm4(wh, sw + lrow * kWRow + (k * 16 + lhalf * 8) * 2);
        ldsm4(wl, sw + kWHalf + lrow * kWRow + (k * 16 + lhalf * 8) * 2);
#pragma unroll
        for (int n2 = 0; n2 < NT / 2; ++n2) {
          uint32_t bv[4];
          ldsm4t(bv, sv + buf * kVBytes + swz<VC>(k * 16 + lrow, warp * NT + 2 * n2 + lhalf));
          mma16816(o[2 * n2], wh[0], wh[1], wh[2], wh[3], bv[0], bv[1]);
          mma16816(o[2 * n2 + 1], wh[0], wh[1], wh[2], wh[3], bv[2], bv[3]);
          mma16816(o[2 * n2], wl[0], wl[1], wl[2], wl[3], bv[0], bv[1]);
          mma16816(o[2 * n2 + 1], wl[0], wl[1], wl[2], wl[3], bv[2], bv[3]);
        }
      }
    }
  }
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = r0 + (e >> 1) * 8, c = (warp * NT + n) * 8 + cq + (e & 1);
      if (h < rep && c < a.V) os[h * a.V + c] = o[n][e];
    }
  __syncthreads();
  const int n = rep * a.V;
  if (a.splits > 1) tc::cluster_sync();
  // every CTA of the cluster finishes a share of the outputs, adding the splits in order
  for (int e = tid + split * kStepThreads; e < n; e += kStepThreads * a.splits) {
    float v = os[e];
    if (a.splits > 1) {
      const uint32_t local = (uint32_t)__cvta_generic_to_shared(&os[e]);
      v = 0.f;
      for (int p = 0; p < a.splits; ++p) v += tc::ld_dsmem_f32(tc::map_to_cta(local, (uint32_t)p));
    }
    a.out[(long long)b * a.ldo + (long long)u * n + e] = us::f2bf(v);
  }
  if (u == 0 && split == 0)
    for (long long c = (long long)H * a.V + tid; c < a.ldo; c += kStepThreads)
      a.out[(long long)b * a.ldo + c] = us::f2bf(0.f);
  if (a.splits > 1) tc::cluster_sync();        // nobody leaves while its sums may still be read
}

template <int NK, int VP>
int launch_apply(const StepArgs& a, cudaStream_t stream) {
  const int rep = a.H / a.G;
  const size_t smem = 2 * kStepTile * VP * 2 + 2 * (NK * 16 + 16) * kWRow + (size_t)rep * a.V * 4;
  static bool configured = false;
  if (!configured) {
    US_CUDA_CHECK(cudaFuncSetAttribute(head_mix_apply_kernel<NK, VP>,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(48 * 1024)));
    configured = true;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(a.splits, a.G, a.B);
  cfg.blockDim = dim3(kStepThreads);
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
  US_CUDA_CHECK(cudaLaunchKernelEx(&cfg, head_mix_apply_kernel<NK, VP>, a));
  return US_OK;
}

template <int kD8>
int launch_scores(const StepArgs& a, cudaStream_t stream) {
  const int rep = a.H / a.G;
  const size_t smem = (size_t)rep * split_keys(a.cap, a.splits) * 4;
  static bool configured = false;
  if (!configured) {
    US_CUDA_CHECK(cudaFuncSetAttribute(head_mix_scores_kernel<kD8>,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024));
    configured = true;
  }
  US_CUDA_CHECK(us::launch_pdl(head_mix_scores_kernel<kD8>, dim3(a.splits, a.G, a.B),
                               dim3(kStepThreads), smem, stream, a));
  return US_OK;
}

// ------------------------------------------------------------------- tiles --
struct TileArgs {
  const __nv_bfloat16* q;
  const __nv_bfloat16 *kc, *vc;
  const float* talk;
  __nv_bfloat16* out;
  const int *cu, *pos, *page_table;
  long long ldq, ldo;
  int B, H, G, D, V, page, max_pages, size, keep;
  float scale_log2;
  int bufs;                   // key / value buffers (1 or 2)
};

constexpr int kTileThreads = 256;
constexpr int kKeys = 16;             // keys per step
constexpr int kOutHeads = 16;         // output heads per CTA (the mixture's 16 rows)
constexpr int kPRow = 16 * kKeys * 2 + 16;   // bytes of a head's probabilities (16 x 16 bf16, padded)

// 16-byte piece of a head's weights that holds row q, keys 8 n .. 8 n + 7 (rows 4 apart take
// opposite halves, so the eight rows of an accumulator store hit different banks; the mixture
// works column by column and needs no order)
__device__ __forceinline__ int ppiece(int q, int n) { return q * 2 + (n ^ ((q >> 2) & 1)); }

// Scores of a warp's HW heads for one step of 16 keys: S[16 rows][16 keys] per head, a lane's
// columns in the two 8-key halves.  Keys are the instruction's columns (row lrow of the tile,
// channel half lhalf); the query fragments come from registers (REG) or shared memory.
template <int HW, int DC, bool REG>
__device__ __forceinline__ void tile_scores(float (&sc)[HW][2][4], const uint32_t (&qf)[HW][DC / 2][4],
                                            uint32_t sq, uint32_t kb, int g0, int H, int rep,
                                            bool one_kv, int lrow, int lhalf) {
  constexpr uint32_t kTileBytes = 16 * DC * 16;
#pragma unroll
  for (int i = 0; i < HW; ++i)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) sc[i][n][e] = 0.f;
#pragma unroll
  for (int k = 0; k < DC / 2; ++k) {
    const uint32_t off = swz<DC>(lrow, 2 * k + lhalf);
    uint32_t bk[4];
    if (one_kv) ldsm4(bk, kb + (uint32_t)(min(g0, H - 1) / rep) * kTileBytes + off);
#pragma unroll
    for (int i = 0; i < HW; ++i) {
      if (!one_kv) ldsm4(bk, kb + (uint32_t)(min(g0 + i, H - 1) / rep) * kTileBytes + off);
      if (REG) {
        mma16816(sc[i][0], qf[i][k][0], qf[i][k][1], qf[i][k][2], qf[i][k][3], bk[0], bk[2]);
        mma16816(sc[i][1], qf[i][k][0], qf[i][k][1], qf[i][k][2], qf[i][k][3], bk[1], bk[3]);
      } else {
        uint32_t aq[4];
        ldsm4(aq, sq + (uint32_t)(g0 + i) * kTileBytes + off);
        mma16816(sc[i][0], aq[0], aq[1], aq[2], aq[3], bk[0], bk[2]);
        mma16816(sc[i][1], aq[0], aq[1], aq[2], aq[3], bk[1], bk[3]);
      }
    }
  }
}

// HP: heads padded to 8, 16 or 32 (8 warps x HP / 8 heads); DP, VP: head widths padded to 64 or
// 128.  blockIdx.x: query tile, blockIdx.y: group of 16 output heads.
template <int HP, int DP, int VP>
__global__ void __launch_bounds__(kTileThreads, 1) head_mix_tile_kernel(const TileArgs a) {
  US_PDL_PROLOGUE();
  constexpr int HW = HP / 8;                       // score heads per warp
  constexpr int OW = HP >= 16 ? 2 : 1;             // output heads per warp
  constexpr int DC = DP / 8, VC = VP / 8;          // 16-byte pieces per row
  extern __shared__ __align__(1024) uint8_t smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  // the query tile: 16 consecutive rows of one sequence
  int tile = blockIdx.x, s = 0, row0 = 0, nrows = 0;
  for (; s < a.B; ++s) {
    const int lo = a.cu[s], n = a.cu[s + 1] - lo, t = (n + 15) >> 4;
    if (tile < t) {
      row0 = lo + tile * 16;
      nrows = min(16, lo + n - row0);
      break;
    }
    tile -= t;
  }
  if (nrows == 0) return;
  const int rep = a.H / a.G;
  const int h_out0 = blockIdx.y * kOutHeads;
  const int n_out = min(kOutHeads, a.H - h_out0);
  const int u_lo = h_out0 / rep, u_n = (h_out0 + n_out - 1) / rep - u_lo + 1;   // value heads needed
  const uint32_t sq = tc::smem_u32(smem);                      // [HP][16][DC]
  const uint32_t sk = sq + HP * 16 * DP * 2;                   // bufs x [G][16][DC]
  const uint32_t k_bytes = (uint32_t)a.G * kKeys * DP * 2;
  const uint32_t sv = sk + a.bufs * k_bytes;                   // bufs x [u_n][16][VC]
  const uint32_t v_bytes = (uint32_t)u_n * kKeys * VP * 2;
  const uint32_t sp = sv + a.bufs * v_bytes;                        // [2: hi, lo][HP16][kPRow]
  constexpr int HK = HP < 16 ? 16 : HP;                        // mixture's inner extent
  const uint32_t p_half = HK * kPRow;
  // queries (heads past H, rows past the tile and channels past D are zero)
  for (int e = tid; e < HP * 16 * DC; e += kTileThreads) {
    const int h = e / (16 * DC), r = (e / DC) & 15, c = e & (DC - 1);
    const uint32_t dst = sq + h * 16 * DP * 2 + swz<DC>(r, c);
    if (h < a.H && r < nrows && c * 8 < a.D)
      cp16(dst, a.q + (long long)(row0 + r) * a.ldq + (long long)h * a.D + c * 8);
    else
      asm volatile("st.shared.v4.u32 [%0], {%1,%1,%1,%1};" ::"r"(dst), "r"(0) : "memory");
  }
  if constexpr (HP < 16) {        // inner rows without a head
    for (int e = tid; e < 2 * (16 - HP) * kPRow / 4; e += kTileThreads) {
      const int half = e / ((16 - HP) * kPRow / 4), x = e - half * ((16 - HP) * kPRow / 4);
      asm volatile("st.shared.u32 [%0], %1;" ::"r"(sp + half * p_half + HP * kPRow + x * 4), "r"(0) : "memory");
    }
  }
  const int p0 = a.pos[row0], p1 = p0 + nrows - 1;
  // keys of the tile: [0, keep) then [lo, p1], or one run from 0 when they meet
  int lo = a.size > 0 ? max(0, p0 - a.size + 1) : 0;
  int kept = max(a.keep, 0);
  if (kept >= lo) { kept = 0; lo = 0; }
  const int kt = (kept + kKeys - 1) / kKeys, steps = kt + (p1 - lo + kKeys) / kKeys;
  const int* pt = a.page_table + (long long)s * a.max_pages;
  const int page_shift = (a.page & (a.page - 1)) == 0 ? __ffs(a.page) - 1 : -1;
  auto slot_of = [&](int key) -> long long {
    const int p = page_shift >= 0 ? key >> page_shift : key / a.page;
    return (long long)pt[p] * a.page + (key - p * a.page);
  };
  auto first_key = [&](int st) { return st < kt ? st * kKeys : lo + (st - kt) * kKeys; };
  auto end_key = [&](int st) { return st < kt ? kept : p1 + 1; };
  // a thread fetches piece c of key row r for every (second, fourth) kv head
  auto load = [&](int st, int buf, bool values) {
    const int k0 = first_key(st), k1 = end_key(st);
    {
      const int c = tid & (DC - 1), r = (tid / DC) & (kKeys - 1), key = k0 + r;
      constexpr int kStride = kTileThreads / (kKeys * DC);
      uint32_t dst = sk + buf * k_bytes + swz<DC>(r, c) + (tid / (kKeys * DC)) * (kKeys * DP * 2);
      const bool ok = key < k1 && c * 8 < a.D;
      const __nv_bfloat16* src = a.kc;
      if (ok) src += (slot_of(key) * a.G + tid / (kKeys * DC)) * a.D + c * 8;
      for (int u = tid / (kKeys * DC); u < a.G; u += kStride) {
        if (ok) cp16(dst, src);
        else asm volatile("st.shared.v4.u32 [%0], {%1,%1,%1,%1};" ::"r"(dst), "r"(0) : "memory");
        dst += kStride * kKeys * DP * 2;
        src += kStride * a.D;
      }
    }
    if (values) {
      const int c = tid & (VC - 1), r = (tid / VC) & (kKeys - 1), key = k0 + r;
      constexpr int kStride = kTileThreads / (kKeys * VC);
      uint32_t dst = sv + buf * v_bytes + swz<VC>(r, c) + (tid / (kKeys * VC)) * (kKeys * VP * 2);
      const bool ok = key < k1 && c * 8 < a.V;
      const __nv_bfloat16* src = a.vc;
      if (ok) src += (slot_of(key) * a.G + u_lo + tid / (kKeys * VC)) * a.V + c * 8;
      for (int u = tid / (kKeys * VC); u < u_n; u += kStride) {
        if (ok) cp16(dst, src);
        else asm volatile("st.shared.v4.u32 [%0], {%1,%1,%1,%1};" ::"r"(dst), "r"(0) : "memory");
        dst += kStride * kKeys * VP * 2;
        src += kStride * a.V;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int lrow = lane & 15, lhalf = lane >> 4;     // ldmatrix row / 8-column half of this lane
  const int r0 = lane >> 2, cq = (lane & 3) * 2;     // accumulator row and first column
  const int g0 = warp * HW;
  const bool one_kv = min(g0, a.H - 1) / rep == min(g0 + HW - 1, a.H - 1) / rep;
  // bit n * 4 + e: row r0 (+8) of the tile sees the key behind accumulator element (n, e)
  auto seen_bits = [&](int st) -> uint32_t {
    const int k0 = first_key(st), k1 = end_key(st);
    // a step every row sees whole: nothing to test
    if (k0 + kKeys <= k1 && k0 + kKeys - 1 <= p0 &&
        (a.size <= 0 || p0 + 15 - k0 < a.size || k0 + kKeys <= a.keep)) return 0xffu;
    uint32_t bits = 0;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = p0 + r0 + (e >> 1) * 8, j = k0 + n * 8 + cq + (e & 1);
        if (j < k1 && j <= i && (a.size <= 0 || i - j < a.size || j < a.keep)) bits |= 1u << (n * 4 + e);
      }
    return bits;
  };
  // ---- first sweep: maximum and sum of every (row, head), in the log2 domain ----
  float mx[HW][2], sum[HW][2];
#pragma unroll
  for (int i = 0; i < HW; ++i) {
    mx[i][0] = mx[i][1] = -INFINITY;
    sum[i][0] = sum[i][1] = 0.f;
  }
  // A step's keys (and values) are fetched while the step before computes, into the other
  // buffer; with one buffer (shapes whose tiles do not fit twice) they are fetched in between.
  const bool two = a.bufs == 2;
  auto next_step = [&](int st, bool values) -> int {
    if (!two) {
      __syncthreads();                      // the step before is done with the buffer
      load(st, 0, values);
    } else if (st == 0) {
      __syncthreads();
      load(0, 0, values);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                        // visible to all; everybody has left the step before
    if (two && st + 1 < steps) load(st + 1, (st + 1) & 1, values);
    return two ? st & 1 : 0;
  };
  {
    uint32_t qf[HW][DC / 2][4];             // the queries stay in registers during this sweep
    for (int st = 0; st < steps; ++st) {
      const int buf = next_step(st, false);
      if (st == 0) {
#pragma unroll
        for (int i = 0; i < HW; ++i)
#pragma unroll
          for (int k = 0; k < DC / 2; ++k)
            ldsm4(qf[i][k], sq + (g0 + i) * 16 * DP * 2 + swz<DC>(lrow, 2 * k + lhalf));
      }
      float sc[HW][2][4];
      tile_scores<HW, DC, true>(sc, qf, sq, sk + buf * k_bytes, g0, a.H, rep, one_kv, lrow, lhalf);
      const uint32_t bits = seen_bits(st);
#pragma unroll
      for (int i = 0; i < HW; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          float v[4], m = mx[i][r];
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int n = x >> 1, e = r * 2 + (x & 1);
            v[x] = (bits >> (n * 4 + e)) & 1u ? sc[i][n][e] * a.scale_log2 : -INFINITY;
            m = fmaxf(m, v[x]);
          }
          const float base = m == -INFINITY ? 0.f : m;      // nothing seen yet: every term is zero
          float l = sum[i][r] * ex2(mx[i][r] - base);
#pragma unroll
          for (int x = 0; x < 4; ++x) l += ex2(v[x] - base);
          sum[i][r] = l;
          mx[i][r] = m;
        }
    }
  }
#pragma unroll
  for (int i = 0; i < HW; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        const float m2 = __shfl_xor_sync(0xffffffffu, mx[i][r], o);
        const float l2 = __shfl_xor_sync(0xffffffffu, sum[i][r], o);
        const float m = fmaxf(mx[i][r], m2);
        if (m != -INFINITY) sum[i][r] = sum[i][r] * ex2(mx[i][r] - m) + l2 * ex2(m2 - m);
        mx[i][r] = m;
      }
      sum[i][r] = sum[i][r] > 0.f ? 1.f / sum[i][r] : 0.f;
    }
  // ---- the mixture's rows T[h_out0 + 0..15][g] as operand fragments ----
  uint32_t tf[HK / 16][4];
#pragma unroll
  for (int k = 0; k < HK / 16; ++k)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = r0 + (e & 1) * 8, g = k * 16 + cq + (e >> 1) * 8;
      const float* t = a.talk + (long long)(h_out0 + h) * a.H + g;
      tf[k][e] = pack_bf(h < n_out && g < a.H ? t[0] : 0.f, h < n_out && g + 1 < a.H ? t[1] : 0.f);
    }
  float o[OW][VP / 8][4];
#pragma unroll
  for (int i = 0; i < OW; ++i)
#pragma unroll
    for (int n = 0; n < VP / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[i][n][e] = 0.f;
  // ---- second sweep ----
  for (int st = 0; st < steps; ++st) {
    const int buf = next_step(st, true);    // (the step before has read its mixed weights)
    {
      float sc[HW][2][4];
      uint32_t none[HW][DC / 2][4];
      tile_scores<HW, DC, false>(sc, none, sq, sk + buf * k_bytes, g0, a.H, rep, one_kv, lrow, lhalf);
      const uint32_t bits = seen_bits(st);
#pragma unroll
      for (int i = 0; i < HW; ++i)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int g = g0 + i, b0 = n * 4 + r * 2;
            float x = ex2(sc[i][n][r * 2] * a.scale_log2 - mx[i][r]) * sum[i][r];
            float y = ex2(sc[i][n][r * 2 + 1] * a.scale_log2 - mx[i][r]) * sum[i][r];
            if (!((bits >> b0) & 1u) || g >= a.H) x = 0.f;
            if (!((bits >> (b0 + 1)) & 1u) || g >= a.H) y = 0.f;
            uint32_t hi, low;
            split_bf(x, y, hi, low);
            const uint32_t dst = sp + g * kPRow + ppiece(r0 + r * 8, n) * 16 + cq * 2;
            asm volatile("st.shared.u32 [%0], %1;" ::"r"(dst), "r"(hi) : "memory");
            asm volatile("st.shared.u32 [%0], %1;" ::"r"(dst + p_half), "r"(low) : "memory");
          }
    }
    __syncthreads();
    // mixture: the warp's 32 columns (2 query rows x 16 keys) of all heads, written back in place
    {
      float w[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) w[n][e] = 0.f;
#pragma unroll
      for (int k = 0; k < HK / 16; ++k)
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int n2 = 0; n2 < 2; ++n2) {
            uint32_t bp[4];
            ldsm4t(bp, sp + part * p_half + (k * 16 + lrow) * kPRow + (warp * 32 + n2 * 16 + lhalf * 8) * 2);
            mma16816(w[n2 * 2], tf[k][0], tf[k][1], tf[k][2], tf[k][3], bp[0], bp[1]);
            mma16816(w[n2 * 2 + 1], tf[k][0], tf[k][1], tf[k][2], tf[k][3], bp[2], bp[3]);
          }
      __syncwarp();
#pragma unroll
      for (int n = 0; n < 4; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          if (HP < 16 && r == 1) continue;
          uint32_t hi, low;
          split_bf(w[n][r * 2], w[n][r * 2 + 1], hi, low);
          const uint32_t dst = sp + (r0 + r * 8) * kPRow + (warp * 32 + n * 8 + cq) * 2;
          asm volatile("st.shared.u32 [%0], %1;" ::"r"(dst), "r"(hi) : "memory");
          asm volatile("st.shared.u32 [%0], %1;" ::"r"(dst + p_half), "r"(low) : "memory");
        }
    }
    __syncthreads();
    // value product of the warp's output heads
#pragma unroll
    for (int i = 0; i < OW; ++i) {
      const int h = warp * OW + i;
      if (h >= n_out) break;
      uint32_t wh[4], wl[4];
      ldsm4(wh, sp + h * kPRow + ppiece(lrow, lhalf) * 16);
      ldsm4(wl, sp + p_half + h * kPRow + ppiece(lrow, lhalf) * 16);
      const uint32_t vb = sv + buf * v_bytes + ((h_out0 + h) / rep - u_lo) * kKeys * VP * 2;
#pragma unroll
      for (int n2 = 0; n2 < VC / 2; ++n2) {
        uint32_t bv[4];
        ldsm4t(bv, vb + swz<VC>(lrow, 2 * n2 + lhalf));
        mma16816(o[i][2 * n2], wh[0], wh[1], wh[2], wh[3], bv[0], bv[1]);
        mma16816(o[i][2 * n2 + 1], wh[0], wh[1], wh[2], wh[3], bv[2], bv[3]);
        mma16816(o[i][2 * n2], wl[0], wl[1], wl[2], wl[3], bv[0], bv[1]);
        mma16816(o[i][2 * n2 + 1], wl[0], wl[1], wl[2], wl[3], bv[2], bv[3]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < OW; ++i) {
    const int h = warp * OW + i;
    if (h >= n_out) break;
#pragma unroll
    for (int n = 0; n < VP / 8; ++n)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int c = n * 8 + cq, row = r0 + r * 8;
        if (row < nrows && c < a.V)
          *reinterpret_cast<uint32_t*>(a.out + (long long)(row0 + row) * a.ldo + (long long)(h_out0 + h) * a.V + c) =
              pack_bf(o[i][n][r * 2], o[i][n][r * 2 + 1]);
      }
  }
  if (blockIdx.y == 0)
    for (int r = 0; r < nrows; ++r)
      for (long long c = (long long)a.H * a.V + tid; c < a.ldo; c += kTileThreads)
        a.out[(long long)(row0 + r) * a.ldo + c] = us::f2bf(0.f);
}

template <int HP, int DP, int VP>
int launch_tile(TileArgs a, int tiles, cudaStream_t stream) {
  const int rep = a.H / a.G;
  int u_n = 1;
  for (int h0 = 0; h0 < a.H; h0 += kOutHeads) {
    const int last = (a.H < h0 + kOutHeads ? a.H : h0 + kOutHeads) - 1;
    const int n = last / rep - h0 / rep + 1;
    u_n = n > u_n ? n : u_n;
  }
  const size_t fixed = (size_t)HP * 16 * DP * 2 + 2 * (size_t)(HP < 16 ? 16 : HP) * kPRow;
  const size_t tile = (size_t)a.G * kKeys * DP * 2 + (size_t)u_n * kKeys * VP * 2;
  a.bufs = fixed + 2 * tile <= 227 * 1024 ? 2 : 1;
  const size_t smem = fixed + a.bufs * tile;
  if (smem > 227 * 1024) return US_ERR_LIMIT;
  static bool configured = false;
  if (!configured) {
    US_CUDA_CHECK(cudaFuncSetAttribute(head_mix_tile_kernel<HP, DP, VP>,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    configured = true;
  }
  US_CUDA_CHECK(us::launch_pdl(head_mix_tile_kernel<HP, DP, VP>,
                               dim3(tiles, (a.H + kOutHeads - 1) / kOutHeads), dim3(kTileThreads), smem,
                               stream, a));
  return US_OK;
}

}  // namespace

// Bytes of scratch of the decode form for rows whose key lists hold at most `cap` keys.
US_API long long us_head_mix_decode_scratch(int B, int H, int cap, int splits) {
  return 4LL * B * H * ((long long)cap + 2LL * splits);
}

// One bf16 row per sequence; US_ERR_UNSUPPORTED / US_ERR_LIMIT for shapes of the row form.
US_API int us_head_mix_decode(const void* q, const void* kc, const void* vc, const float* talk,
                              void* out, const int* pos, const int* page_table, const int* seq_lens,
                              void* scratch, long long ldq, long long ldo, int B, int H, int G, int D,
                              int V, int page, int max_pages, int size, int keep, int cap, int splits,
                              float scale, void* stream_) {
  US_REQUIRE(q && kc && vc && talk && out && pos && page_table && seq_lens && scratch && B >= 1);
  US_REQUIRE(H >= 1 && G >= 1 && H % G == 0 && page >= 1 && cap >= 1 && splits >= 1 && splits <= 8);
  US_REQUIRE(ldo >= (long long)H * V && ((uintptr_t)q % 16) == 0 && ((uintptr_t)kc % 16) == 0 &&
             ((uintptr_t)vc % 16) == 0 && (ldq % 8) == 0);
  const int rep = H / G;
  if ((D % 8) || D > 256 || (V % 8) || V > 128 || rep > 16 || H > 64 || (cap % 2) || B > 65535)
    return US_ERR_UNSUPPORTED;
  if ((long long)rep * split_keys(cap, splits) * 4 > 100 * 1024) return US_ERR_LIMIT;
  StepArgs a{(const __nv_bfloat16*)q, (const __nv_bfloat16*)kc, (const __nv_bfloat16*)vc, talk,
             (__nv_bfloat16*)out, (float*)scratch, (float*)scratch + (long long)B * H * cap, pos,
             page_table, seq_lens, ldq, ldo, B, H, G, D, V, page, max_pages, size, keep, cap, splits,
             scale};
  cudaStream_t stream = (cudaStream_t)stream_;
  int rc = D <= 64 ? launch_scores<2>(a, stream) : D <= 128 ? launch_scores<4>(a, stream)
                                                            : launch_scores<8>(a, stream);
  if (rc) return rc;
#define US_HM(NK) \
  return V <= 64 ? launch_apply<NK, 64>(a, stream) : launch_apply<NK, 128>(a, stream);
  if (H <= 16) { US_HM(1) }
  if (H <= 32) { US_HM(2) }
  US_HM(4)
#undef US_HM
}

// bf16 rows of packed sequences; `rows` bounds the tiles.
US_API int us_head_mix_prefill(const void* q, const void* kc, const void* vc, const float* talk,
                               void* out, const int* cu, const int* pos, const int* page_table,
                               long long ldq, long long ldo, int rows, int B, int H, int G, int D,
                               int V, int page, int max_pages, int size, int keep, float scale,
                               void* stream_) {
  US_REQUIRE(q && kc && vc && talk && out && cu && pos && page_table && rows >= 1 && B >= 1);
  US_REQUIRE(H >= 1 && G >= 1 && H % G == 0 && page >= 1 && ldo >= (long long)H * V);
  US_REQUIRE(((uintptr_t)q % 16) == 0 && ((uintptr_t)kc % 16) == 0 && ((uintptr_t)vc % 16) == 0 &&
             (ldq % 8) == 0 && (ldo % 2) == 0);
  if ((D % 8) || D > 128 || (V % 8) || V > 128 || H > 32) return US_ERR_UNSUPPORTED;
  TileArgs a{(const __nv_bfloat16*)q, (const __nv_bfloat16*)kc, (const __nv_bfloat16*)vc, talk,
             (__nv_bfloat16*)out, cu, pos, page_table, ldq, ldo, B, H, G, D, V, page, max_pages, size,
             keep, scale * 1.4426950408889634f, 2};
  cudaStream_t stream = (cudaStream_t)stream_;
  const int tiles = rows / 16 + B;
#define US_HT2(HP, DP) \
  return V <= 64 ? launch_tile<HP, DP, 64>(a, tiles, stream) : launch_tile<HP, DP, 128>(a, tiles, stream);
#define US_HT(HP) \
  if (D <= 64) { US_HT2(HP, 64) } else { US_HT2(HP, 128) }
  if (H <= 8) { US_HT(8) }
  if (H <= 16) { US_HT(16) }
  US_HT(32)
#undef US_HT
#undef US_HT2
}

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
