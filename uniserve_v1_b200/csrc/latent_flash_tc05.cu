// Latent attention for prompts (see latent_attn.cu), bf16: keys and values of the tokens in view are
// formed per head (one product with the stacked W_uk | W_uv) and a windowed causal flash kernel on
// tcgen05 runs over them.
//
//   us_latent_gather    the latents and rotated parts that a batch's prompts see, from their pages
//                       into packed rows (sequence by sequence, oldest first)
//   us_latent_flash     score = q_unrotated . k_head + q_rotated . k_shared, window, softmax, values
//   us_window_flash     score = q . k, grouped heads, window, softmax with a sink, values
//   us_sigmoid_flash    the same with a key's weight the sigmoid of its capped and shifted score (no softmax)
//
// The flash kernel is the two-tile scheme of flash_attn2_tc05.cu with unlike operands: a CTA owns 256
// query rows of one (sequence, head) as tiles A and B; keys come in blocks of 128 as one or two
// 64-channel slabs of the head's own keys and, in the latent form, one slab of the rotated part that
// all heads share.
// Where 192-wide keys leave no room for two value stages there is one; the block of values is then
// fetched while the tensor pipe forms the next scores.  Blocks outside a tile's window are skipped.
// Without a softmax there is neither a maximum nor a sum: weights go straight into the value product, whose
// accumulator is never rescaled.  Every wait is bounded.
#include "include/us_common.cuh"
#include "include/us_flash.cuh"
#include "include/us_mma.cuh"
#include "include/us_tc05.cuh"
#include "include/us_tmap.h"

namespace {

using namespace flash;

constexpr int kBM = 128, kBN = 128;
constexpr int kSlab = 128 * 128;         // bytes of 128 rows x 64 columns
constexpr float kRescaleThreshold = 8.f; // log2 units

// ------------------------------------------------------------------ gather --
struct GatherArgs {
  const __nv_bfloat16 *cp, *rp;          // pages [n, page, ldc], [n, page, ldr]
  int ldc, ldr, page, max_pages;
  __nv_bfloat16 *c, *r;                  // [rows, ldc], [rows, 64]
  int* cu_k;                             // [B + 1]
  const int *cu, *pos, *page_table;
  int B, window, min_rows, rows;
};

// keys that sequence s sees in this batch (0: too few rows, it is served elsewhere) and the first one
__device__ __forceinline__ int seen(const GatherArgs& a, int s, int& first) {
  const int q = a.cu[s + 1] - a.cu[s];
  first = 0;
  if (q < a.min_rows) return 0;
  const int p0 = a.pos[a.cu[s]];
  first = a.window > 0 ? max(0, p0 - a.window + 1) : 0;
  return p0 + q - first;
}

__global__ void __launch_bounds__(256) latent_gather_kernel(const GatherArgs a) {
  US_PDL_PROLOGUE();
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  int at = 0, first = 0, s = 0, n = 0;
  for (; s < a.B; ++s) {
    n = seen(a, s, first);
    if (blockIdx.x == 0 && threadIdx.x == 0) a.cu_k[s] = at;
    if (row < at + n && blockIdx.x != 0) break;
    if (blockIdx.x == 0 && row >= at && row < at + n) {      // block 0 walks on for cu_k
      const int key = first + row - at;
      const long long src = (long long)a.page_table[(long long)s * a.max_pages + key / a.page] * a.page + key % a.page;
      for (int c = lane * 8; c < a.ldc; c += 256)
        *reinterpret_cast<uint4*>(a.c + (long long)row * a.ldc + c) =
            *reinterpret_cast<const uint4*>(a.cp + src * a.ldc + c);
      if (lane < 8)
        *reinterpret_cast<uint4*>(a.r + (long long)row * 64 + lane * 8) =
            lane * 8 < a.ldr ? *reinterpret_cast<const uint4*>(a.rp + src * a.ldr + lane * 8)
                             : make_uint4(0, 0, 0, 0);
    }
    at += n;
  }
  if (blockIdx.x == 0) {
    if (threadIdx.x == 0) a.cu_k[a.B] = at;
    return;
  }
  if (s == a.B || row >= a.rows) return;
  const int key = first + row - at;
  const long long src = (long long)a.page_table[(long long)s * a.max_pages + key / a.page] * a.page + key % a.page;
  for (int c = lane * 8; c < a.ldc; c += 256)
    *reinterpret_cast<uint4*>(a.c + (long long)row * a.ldc + c) =
        *reinterpret_cast<const uint4*>(a.cp + src * a.ldc + c);
  if (lane < 8)
    *reinterpret_cast<uint4*>(a.r + (long long)row * 64 + lane * 8) =
        lane * 8 < a.ldr ? *reinterpret_cast<const uint4*>(a.rp + src * a.ldr + lane * 8)
                         : make_uint4(0, 0, 0, 0);
}

// ------------------------------------------------------------------- flash --
struct FlashArgs {
  const int *cu_q, *cu_k;
  __nv_bfloat16* out;                    // [T, ldo], head h at column h * V
  long long ldo;
  int V, window;
  float scale_log2;
  unsigned int* status;
  int rep;                               // query heads per key / value head
  const float* sink;                     // [H] or null: exp(sink) joins the softmax denominator
  float out_scale;
  // or null: the output times the sigmoid of column h * gate_cols + (column of the head) % gate_cols of
  // the row (gate_cols 1: a logit per head, V: one per column)
  const __nv_bfloat16* gate;
  long long ldg;
  int gate_cols;
  // sigmoid form: z = score * scale * temp / cap, weight = sigmoid(cap * tanh(z) + shift)
  const float *temp, *shift;             // [H]
  float scale, cap;
};

// tanh(z) / z as polynomials in u = z^2 (least maximum error: 1.3e-8 up to |z| = 1/2, 3.8e-8 up to 6/5)
constexpr float kTanhNear = 0.5f, kTanhFar = 1.2f;
__device__ constexpr float kNear[5] = {1.f, -0.33333075046539307f, 0.13324907422065735f, -0.05299423262476921f,
                                       0.017151299864053726f};
__device__ constexpr float kFar[8] = {1.f, -0.3333297073841095f, 0.13327667117118835f, -0.053627558052539825f,
                                      0.020839421078562737f, -0.007092796266078949f, 0.001742084277793765f,
                                      -0.00021388338063843548f};
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kExpMost = 60.f;         // exponents (base 2) up to here keep the product of two sums finite

// Weights of a row's scores, two at a time with one reciprocal: sigmoid(cap tanh(z) + shift), z = score * f.
struct SigWeights {
  float near, far;                       // scores up to here take a polynomial; up to `near` no exponent passes kExpMost
  float f, c, f_shift;                   // exponent (base 2) of the negated argument: c * tanh(score * f) + f_shift
  __device__ __forceinline__ SigWeights(float f_, float cap, float shift)
      : f(f_), c(-cap * kLog2e), f_shift(-shift * kLog2e) {
    near = fminf(kTanhNear, (kExpMost / kLog2e - fabsf(shift)) / cap) / fabsf(f);
    far = kTanhFar / fabsf(f);
  }
  // two exponents -> two weights as bf16
  static __device__ __forceinline__ uint32_t weigh(float x0, float x1) {
    float a0, a1;
    unpack2(add2(pack2(ex2f(x0), ex2f(x1)), pack2(1.f, 1.f)), a0, a1);
    const float r = rcpf(a0 * a1);
    return us::pack_bf(r * a1, r * a0);
  }
  // score * (k_0 + k_1 score^2 + ..) with the factors of score, cap and base in the coefficients
  template <int N, bool kClamp>
  __device__ __forceinline__ void by_polynomial(const uint32_t (&v)[32], uint32_t (&w)[16], const float (&k)[N]) const {
    unsigned long long b[N];
    float at = c * f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      b[i] = pack2(k[i] * at, k[i] * at);
      at *= f * f;
    }
    const unsigned long long sh = pack2(f_shift, f_shift);
#pragma unroll
    for (int i = 0; i < 32; i += 2) {
      const unsigned long long s = pack2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), u = mul2(s, s);
      unsigned long long p = b[N - 1];
#pragma unroll
      for (int e = N - 2; e >= 0; --e) p = fma2(p, u, b[e]);
      float x0, x1;
      unpack2(fma2(s, p, sh), x0, x1);
      w[i >> 1] = kClamp ? weigh(fminf(x0, kExpMost), fminf(x1, kExpMost)) : weigh(x0, x1);
    }
  }
  __device__ __forceinline__ void operator()(const uint32_t (&v)[32], uint32_t (&w)[16]) const {
    float top[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < 32; i += 4)
#pragma unroll
      for (int e = 0; e < 2; ++e)
        top[e] = max3_abs(top[e], __uint_as_float(v[i + 2 * e]), __uint_as_float(v[i + 2 * e + 1]));
    const float most = fmaxf(top[0], top[1]);
    if (__all_sync(0xffffffffu, most <= near)) {
      by_polynomial<5, false>(v, w, {kNear[0], kNear[1], kNear[2], kNear[3], kNear[4]});
    } else if (__all_sync(0xffffffffu, most <= far)) {
      by_polynomial<8, true>(v, w, {kFar[0], kFar[1], kFar[2], kFar[3], kFar[4], kFar[5], kFar[6], kFar[7]});
    } else {
      const float f_e = 2.f * kLog2e * f;    // e^{2 z} = 2^{score f_e}, tanh(z) = 1 - 2 / (e^{2 z} + 1)
#pragma unroll
      for (int i = 0; i < 32; i += 2) {
        const float e0 = ex2f(fminf(__uint_as_float(v[i]) * f_e, kExpMost)) + 1.f;
        const float e1 = ex2f(fminf(__uint_as_float(v[i + 1]) * f_e, kExpMost)) + 1.f;
        const float r = -2.f * rcpf(e0 * e1);
        const float t0 = fmaf(r, e1, 1.f), t1 = fmaf(r, e0, 1.f);
        w[i >> 1] = weigh(fminf(fmaf(t0, c, f_shift), kExpMost), fminf(fmaf(t1, c, f_shift), kExpMost));
      }
    }
  }
};

__device__ __forceinline__ float sigmoid_of(__nv_bfloat16 x) { return 1.f / (1.f + __expf(-us::bf2f(x))); }

// kN: 64-channel slabs of the head's own keys; kR: slabs of the shared part (0 or 1); kDV: value
// width; kVS: value stages; kSig: sigmoid weights.
template <int kN, int kR, int kDV, int kVS, bool kSig>
__global__ void __launch_bounds__(320, 1)
latent_flash_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                    const __grid_constant__ CUtensorMap tmR, const __grid_constant__ CUtensorMap tmV,
                    const FlashArgs a) {
  US_PDL_PROLOGUE();
  constexpr int kS = kN + kR;                    // slabs of a query or key tile
  constexpr int kTile = kS * kSlab, kVTile = kDV / 64 * kSlab;
  const int q_pair = a.window > 0 ? (int)blockIdx.x : (int)gridDim.x - 1 - (int)blockIdx.x;
  const int h = blockIdx.y, hk = h / a.rep, seq = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  constexpr int kTmaWarp = 8, kMmaWarp = 9;
  const int q_start = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_start;
  const int k_start = a.cu_k[seq], kv_len = a.cu_k[seq + 1] - k_start;
  const int q0 = q_pair * 2 * kBM;
  if (q0 >= q_len || kv_len <= 0) return;
  const int shift = kv_len - q_len;              // key <= query + shift
  int jb[2], je[2];                              // key blocks of each tile
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int q0x = q0 + x * kBM;
    jb[x] = a.window > 0 ? max(0, q0x + shift - a.window + 1) / kBN : 0;
    je[x] = q0x < q_len ? (min(kv_len, q0x + kBM + shift) + kBN - 1) / kBN : jb[x];
  }
  const int j_lo = jb[0], nb = max(je[0], je[1]) - j_lo;
#pragma unroll
  for (int x = 0; x < 2; ++x) {                  // from here on relative to the first block
    jb[x] -= j_lo;
    je[x] -= j_lo;
  }

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint8_t* sQ = smem;                            // two tiles
  uint8_t* sK = sQ + 2 * kTile;                  // two stages
  uint8_t* sV = sK + 2 * kTile;                  // kVS stages
  uint64_t* bars = (uint64_t*)(sV + kVS * kVTile);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;    // [2]
  uint64_t* k_empty = bars + 3;   // [2]
  uint64_t* v_full = bars + 5;    // [2]
  uint64_t* v_empty = bars + 7;   // [2]
  uint64_t* s_full = bars + 9;    // [2] per tile
  uint64_t* p_full = bars + 11;   // [2] per tile
  uint64_t* o_full = bars + 13;   // [2] per tile
  uint32_t* tmem_slot = (uint32_t*)(bars + 15);
  volatile uint32_t* abort_flag = tmem_slot + 1;

  if (tid == 0) {
    tc::mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      tc::mbar_init(&k_full[i], 1);
      tc::mbar_init(&k_empty[i], 1);
      tc::mbar_init(&v_full[i], 1);
      tc::mbar_init(&v_empty[i], 1);
      tc::mbar_init(&s_full[i], 1);
      tc::mbar_init(&p_full[i], 128);
      tc::mbar_init(&o_full[i], 1);
    }
    *abort_flag = 0;
    tc::mbar_fence_init();
  }
  if (warp == kMmaWarp) {
    tc::tmem_alloc(tmem_slot, 512);
    tc::tmem_relinquish();
  }
  tc::tc_fence_before_sync();
  __syncthreads();
  tc::tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == kTmaWarp) {
    if (lane == 0) {
      tc::mbar_expect_tx(q_full, 2 * kTile);
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int p = 0; p < kS; ++p)             // rows past the tensor read as zeros
          tc::tma_load_2d(sQ + x * kTile + p * kSlab, &tmQ, q_full, (h * kS + p) * 64,
                          q_start + q0 + x * kBM);
      bool ok = true;
      auto load_k = [&](int j) {
        const int st = j & 1, row = k_start + (j_lo + j) * kBN;
        if (!tc::mbar_wait(&k_empty[st], ((uint32_t)(j >> 1) & 1u) ^ 1u, abort_flag)) return false;
        tc::mbar_expect_tx(&k_full[st], kTile);
#pragma unroll
        for (int p = 0; p < kN; ++p)
          tc::tma_load_2d(sK + st * kTile + p * kSlab, &tmK, &k_full[st], (hk * kN + p) * 64, row);
        if (kR) tc::tma_load_2d(sK + st * kTile + kN * kSlab, &tmR, &k_full[st], 0, row);
        return true;
      };
      auto load_v = [&](int j) {
        const int st = j % kVS, row = k_start + (j_lo + j) * kBN;
        if (!tc::mbar_wait(&v_empty[st], ((uint32_t)(j / kVS) & 1u) ^ 1u, abort_flag)) return false;
        tc::mbar_expect_tx(&v_full[st], kVTile);
#pragma unroll
        for (int p = 0; p < kDV / 64; ++p)
          tc::tma_load_2d(sV + st * kVTile + p * kSlab, &tmV, &v_full[st], hk * kDV + p * 64, row);
        return true;
      };
      ok = load_k(0) && (nb < 2 || load_k(1));
      for (int j = 0; ok && j < nb; ++j) ok = load_v(j) && (j + 2 >= nb || load_k(j + 2));
      if (!ok) {
        us_dev_fail(a.status, US_DEV_TIMEOUT_EMPTY);
        *abort_flag = 1;
      }
    }
  } else if (warp == kMmaWarp) {
    // all 32 lanes, converged; single lanes are elected per instruction
    auto warp_wait = [&](uint64_t* bar, uint32_t parity) -> bool {
      return __all_sync(0xffffffffu, tc::mbar_wait(bar, parity, abort_flag));
    };
    constexpr uint32_t kIdescQK = tc::make_idesc(kBM, kBN, tc::kFmtBF16, tc::kFmtBF16, 0, 0);
    constexpr uint32_t kIdescPV = tc::make_idesc(kBM, kDV, tc::kFmtBF16, tc::kFmtBF16, 0, 1);
    const uint64_t dq = tc::smem_desc_kmajor_sw128(tc::smem_u32(sQ));
    const uint64_t dk = tc::smem_desc_kmajor_sw128(tc::smem_u32(sK));
    const uint64_t dv = tc::smem_desc_mnmajor_sw128(tc::smem_u32(sV), kSlab, 1024);
    const uint32_t q_lo = (uint32_t)dq, k_lo = (uint32_t)dk, v_lo = (uint32_t)dv;
    const uint32_t km_hi = (uint32_t)(dq >> 32), mn_hi = (uint32_t)(dv >> 32);
    auto issue_qk = [&](int x, int j) {
      const uint32_t qa = q_lo + (uint32_t)x * (kTile >> 4);
      const uint32_t kb = k_lo + (uint32_t)(j & 1) * (kTile >> 4);
      const uint32_t s_tmem = tmem_base + (uint32_t)x * kBN;
#pragma unroll
      for (int kk = 0; kk < kS * 4; ++kk) {
        const uint32_t off = (uint32_t)(kk >> 2) * (kSlab >> 4) + 2u * (uint32_t)(kk & 3);
        umma_f16_words(s_tmem, qa + off, km_hi, kb + off, km_hi, kIdescQK, kk != 0);
      }
      umma_commit_elect(&s_full[x]);
    };
    auto issue_pv = [&](int x, int j) {
      const uint32_t vb = v_lo + (uint32_t)(j % kVS) * (kVTile >> 4);
      const uint32_t p_tmem = tmem_base + (uint32_t)x * kBN;
      const uint32_t o_tmem = tmem_base + 256 + (uint32_t)x * kDV;
#pragma unroll
      for (int kk = 0; kk < 8; ++kk)
        umma_f16_ts_words(o_tmem, p_tmem + kk * 8, vb + (uint32_t)kk * (2048 >> 4), mn_hi, kIdescPV,
                          (j != jb[x]) || kk != 0);
      if (j == je[x] - 1) umma_commit_elect(&o_full[x]);
    };
    bool ok = warp_wait(q_full, 0) && warp_wait(&k_full[0], 0);
    if (ok) {
      tc::tc_fence_after_sync();
#pragma unroll
      for (int x = 0; x < 2; ++x)
        if (jb[x] <= 0 && 0 < je[x]) issue_qk(x, 0);
      umma_commit_elect(&k_empty[0]);
    }
    for (int j = 0; ok && j < nb; ++j) {
      ok = warp_wait(&v_full[j % kVS], (uint32_t)(j / kVS) & 1u);
      bool next = false;                         // K(j + 1) is there
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        if (!ok) break;
        if (jb[x] <= j && j < je[x]) {
          ok = warp_wait(&p_full[x], (uint32_t)(j - jb[x]) & 1u);
          if (!ok) break;
          tc::tc_fence_after_sync();
          issue_pv(x, j);
        }
        if (x == 1) umma_commit_elect(&v_empty[j % kVS]);
        if (jb[x] <= j + 1 && j + 1 < je[x]) {
          if (!next) {
            ok = warp_wait(&k_full[(j + 1) & 1], (uint32_t)((j + 1) >> 1) & 1u);
            if (!ok) break;
            tc::tc_fence_after_sync();
            next = true;
          }
          issue_qk(x, j + 1);
        }
      }
      if (ok && j + 1 < nb) umma_commit_elect(&k_empty[(j + 1) & 1]);
    }
    if (!ok && lane == 0) {
      us_dev_fail(a.status, US_DEV_TIMEOUT_FULL);
      *abort_flag = 1;
    }
  } else {
    // ---- softmax: warpgroup per tile, thread = query row ----
    const int x = warp >> 2;
    const int r = (warp & 3) * 32 + lane;
    const uint32_t lane_addr = ((uint32_t)((warp & 3) * 32) << 16);
    const uint32_t s_tmem = tmem_base + (uint32_t)x * kBN + lane_addr;
    const uint32_t o_tmem = tmem_base + 256 + (uint32_t)x * kDV + lane_addr;
    const int q_idx = q0 + x * kBM + r;
    const int j0 = x ? jb[1] : jb[0], j1 = x ? je[1] : je[0];
    float m_used = -INFINITY, l_sum = 0.f;
    const SigWeights weights(kSig ? a.scale * a.temp[h] / a.cap : 1.f, kSig ? a.cap : 1.f, kSig ? a.shift[h] : 0.f);
    bool ok = true;
    for (int j = j0; j < j1; ++j) {
      ok = __all_sync(0xffffffffu, tc::mbar_wait(&s_full[x], (uint32_t)(j - j0) & 1u, abort_flag));
      if (!ok) break;
      tc::tc_fence_after_sync();
      // keys of this block the row sees: [low, lim)
      const int kbase = (j_lo + j) * kBN, q_rel = q_idx + shift;
      const int lim = min(kv_len, q_rel + 1) - kbase;
      const int low = a.window > 0 ? q_rel - a.window + 1 - kbase : 0;
      if constexpr (kSig) {
        // 32 columns at a time, the next ones on their way; their weights go where scores have been read
        uint32_t v[2][32];
        tc::tmem_ld32(s_tmem, v[0]);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          tc::tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) asm volatile("" : "+r"(v[c & 1][i]));     // not before the wait
          if (c < 3) tc::tmem_ld32(s_tmem + 32 * (c + 1), v[(c + 1) & 1]);
          uint32_t pk[16];
          weights(v[c & 1], pk);
          const int l0 = low - 32 * c, l1 = lim - 32 * c;
          if (l1 < 32 || l0 > 0) {
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              if (i >= l1 || i < l0) pk[i >> 1] &= 0xffff0000u;
              if (i + 1 >= l1 || i + 1 < l0) pk[i >> 1] &= 0x0000ffffu;
            }
          }
          tc::tmem_st16(s_tmem + 16 * c, pk);
        }
        tc::tmem_st_wait();
        tc::tc_fence_before_sync();
        tc::mbar_arrive(&p_full[x]);
        continue;
      }
      uint32_t v[kBN];
#pragma unroll
      for (int c = 0; c < 4; ++c)
        tc::tmem_ld32(s_tmem + 32 * c, *reinterpret_cast<uint32_t(*)[32]>(v + 32 * c));
      tc::tmem_ld_wait();
      if (lim < kBN || low > 0) {
#pragma unroll
        for (int i = 0; i < kBN; ++i)
          if (i >= lim || i < low) v[i] = 0xff800000u;
      }
      float mxs[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < 32; i += 2)
#pragma unroll
        for (int c = 0; c < 4; ++c)
          mxs[c] = max3(mxs[c], __uint_as_float(v[32 * c + i]), __uint_as_float(v[32 * c + i + 1]));
      const float mx = fmaxf(fmaxf(mxs[0], mxs[1]), fmaxf(mxs[2], mxs[3]));
      const float m_new = fmaxf(m_used, mx * a.scale_log2);
      const bool grow = m_new - m_used > kRescaleThreshold;
      if (__any_sync(0xffffffffu, grow || (m_used == -INFINITY && m_new > -INFINITY))) {
        const float alpha = (m_used == -INFINITY) ? 0.f : ex2f(m_used - m_new);
        if (j > j0) {
          // O is stable: this block's scores were issued after the previous block's value product
          // by the same thread, and the commit that filled s_full covers both
#pragma unroll 1
          for (int c = 0; c < kDV; c += 32) {
            uint32_t w[32];
            tc::tmem_ld32(o_tmem + c, w);
            tc::tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) w[i] = __float_as_uint(__uint_as_float(w[i]) * alpha);
            tc::tmem_st32(o_tmem + c, w);
          }
        }
        l_sum *= alpha;
        m_used = m_new;
      }
      const float neg_m = (m_used == -INFINITY) ? 0.f : -m_used;
      const unsigned long long nm2 = pack2(neg_m, neg_m), sc2 = pack2(a.scale_log2, a.scale_log2);
      unsigned long long ls[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) ls[c] = pack2(0.f, 0.f);
      uint32_t pk[kBN / 2];
#pragma unroll
      for (int i = 0; i < 32; i += 2)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          float t0, t1;
          unpack2(fma2(pack2(__uint_as_float(v[32 * c + i]), __uint_as_float(v[32 * c + i + 1])), sc2, nm2), t0, t1);
          t0 = ex2f(t0);
          t1 = ex2f(t1);
          ls[c] = add2(ls[c], pack2(t0, t1));
          pk[16 * c + (i >> 1)] = us::pack_bf(t0, t1);
        }
      float s0, s1;
      unpack2(add2(add2(ls[0], ls[1]), add2(ls[2], ls[3])), s0, s1);
      l_sum += s0 + s1;
      // P (packed pairs) replaces the first half of S, which is in registers by now
#pragma unroll
      for (int c = 0; c < 2; ++c)
        tc::tmem_st32(s_tmem + 32 * c, *reinterpret_cast<const uint32_t(*)[32]>(pk + 32 * c));
      tc::tmem_st_wait();
      tc::tc_fence_before_sync();
      tc::mbar_arrive(&p_full[x]);
    }
    if (j1 > j0) {
      const bool row_ok = q_idx < q_len, wide = ((a.V | (int)a.ldo) & 7) == 0;
      const long long row = q_start + q_idx;
      // a gate of every column: fetched in 16-byte pieces while the last value product runs
      const bool columns = a.gate && a.gate_cols > 1;
      const bool pieces = columns && wide && (a.ldg & 7) == 0 && ((uintptr_t)a.gate & 15) == 0;
      const __nv_bfloat16* grow = a.gate ? a.gate + row * a.ldg + (long long)h * a.gate_cols : nullptr;
      uint4 gp[kDV / 8];
      if (pieces) {
#pragma unroll
        for (int i = 0; i < kDV / 8; ++i)
          if (row_ok && i * 8 < a.V) gp[i] = __ldg(reinterpret_cast<const uint4*>(grow) + i);
      }
      if (ok && tc::mbar_wait(&o_full[x], 0, abort_flag)) {
        tc::tc_fence_after_sync();
        if (a.sink && l_sum > 0.f) l_sum += ex2f(a.sink[h] * kLog2e - m_used);
        float inv = kSig ? a.out_scale : l_sum > 0.f ? a.out_scale / l_sum : 0.f;
        if (a.gate && !columns && row_ok) inv *= sigmoid_of(*grow);
        __nv_bfloat16* orow = a.out + row * a.ldo + (long long)h * a.V;
        if (pieces) {
#pragma unroll
          for (int c = 0; c < kDV; c += 32) {
            uint32_t w[32];
            tc::tmem_ld32(o_tmem + c, w);
            tc::tmem_ld_wait();
            if (!row_ok) continue;
#pragma unroll
            for (int q4 = 0; q4 < 4; ++q4) {
              if (c + q4 * 8 >= a.V) continue;
              us::Pack16 o, g;
              g.u = gp[c / 8 + q4];
#pragma unroll
              for (int i = 0; i < 8; i += 2) {         // two sigmoids with one reciprocal
                const float g0 = ex2f(fminf(us::bf2f(g.b[i]) * -kLog2e, kExpMost)) + 1.f;
                const float g1 = ex2f(fminf(us::bf2f(g.b[i + 1]) * -kLog2e, kExpMost)) + 1.f;
                const float r = inv * rcpf(g0 * g1);
                o.b[i] = us::f2bf(__uint_as_float(w[q4 * 8 + i]) * (r * g1));
                o.b[i + 1] = us::f2bf(__uint_as_float(w[q4 * 8 + i + 1]) * (r * g0));
              }
              *reinterpret_cast<uint4*>(orow + c + q4 * 8) = o.u;
            }
          }
        } else {
#pragma unroll 1
          for (int c = 0; c < kDV; c += 32) {
            uint32_t w[32];
            tc::tmem_ld32(o_tmem + c, w);
            tc::tmem_ld_wait();
            if (!row_ok) continue;
#pragma unroll
            for (int q4 = 0; q4 < 4; ++q4) {
              us::Pack16 o;
#pragma unroll
              for (int i = 0; i < 8; ++i) {
                float f = __uint_as_float(w[q4 * 8 + i]) * inv;
                if (columns && c + q4 * 8 + i < a.V) f *= sigmoid_of(grow[c + q4 * 8 + i]);
                o.b[i] = us::f2bf(f);
              }
              if (wide) {
                if (c + q4 * 8 < a.V) *reinterpret_cast<uint4*>(orow + c + q4 * 8) = o.u;
              } else {
#pragma unroll
                for (int i = 0; i < 8; ++i)
                  if (c + q4 * 8 + i < a.V) orow[c + q4 * 8 + i] = o.b[i];
              }
            }
          }
        }
      } else {
        us_dev_fail(a.status, US_DEV_TIMEOUT_ACC);
      }
    }
  }
  tc::tc_fence_before_sync();
  __syncthreads();
  if (warp == kMmaWarp) {
    __syncwarp();
    tc::tmem_dealloc(tmem_base, 512);
  }
}

template <int kN, int kR, int kDV, int kVS, bool kSig = false>
int launch_flash(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmR,
                 const CUtensorMap& tmV, const FlashArgs& a, dim3 grid, cudaStream_t stream) {
  constexpr size_t smem = (size_t)4 * (kN + kR) * kSlab + (size_t)kVS * (kDV / 64) * kSlab + 17 * 8 + 1024;
  static_assert(smem <= 227 * 1024, "shared memory of a CTA");
  static bool configured = false;
  if (!configured) {
    US_CUDA_CHECK(cudaFuncSetAttribute(latent_flash_kernel<kN, kR, kDV, kVS, kSig>,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = true;
  }
  US_CUDA_CHECK(us::launch_pdl(latent_flash_kernel<kN, kR, kDV, kVS, kSig>, grid, dim3(320), smem, stream, tmQ,
                               tmK, tmR, tmV, a));
  return US_OK;
}

}  // namespace

// Packs what sequences of at least `min_rows` rows see (window 0: everything) into c [rows, ldc] and
// r [rows, 64]; writes their offsets to cu_k.  `rows` is their number, known to the host.
US_API int us_latent_gather(const void* cpages, int ldc, const void* rpages, int ldr, void* c, void* r,
                            int* cu_k, const int* cu, const int* pos, const int* page_table, int B,
                            int page, int max_pages, int window, int min_rows, int rows,
                            void* stream_) {
  US_REQUIRE(cpages && rpages && c && r && cu_k && cu && pos && page_table && B >= 1 && page >= 1 &&
             rows >= 1 && min_rows >= 1 && (ldc % 8) == 0 && (ldr % 8) == 0 && ldr <= 64);
  GatherArgs a{(const __nv_bfloat16*)cpages, (const __nv_bfloat16*)rpages, ldc, ldr, page, max_pages,
               (__nv_bfloat16*)c, (__nv_bfloat16*)r, cu_k, cu, pos, page_table, B, window, min_rows, rows};
  US_CUDA_CHECK(us::launch_pdl(latent_gather_kernel, dim3(us::ceil_div(rows, 8)), dim3(256), 0,
                               (cudaStream_t)stream_, a));
  return US_OK;
}

// q [Tq, H (slabs + 1) 64] rows at ldq: per head its unrotated channels in `slabs` slabs of 64, then the
// rotated ones; kv [Tk, H slabs 64 | H dv] rows at ldkv; r [Tk, 64]; V <= dv output columns per head.
// gate [Tq, H V] rows at ldg, or null: the output times its sigmoid.  Sequences without keys (cu_k) are left alone.
US_API int us_latent_flash(const void* q, long long ldq, const void* kv, long long ldkv, const void* r,
                           void* out, long long ldo, const int* cu_q, const int* cu_k, int n_seqs,
                           int Tq, int Tk, int H, int slabs, int dv, int V, int max_q, int window,
                           float scale, const void* gate, long long ldg, void* stream_) {
  US_REQUIRE(q && kv && r && out && cu_q && cu_k && n_seqs >= 1 && Tq >= 1 && Tk >= 1 && H >= 1 &&
             max_q >= 1 && V >= 1 && V <= dv);
  US_REQUIRE((ldq % 8) == 0 && (ldkv % 8) == 0 && ((uintptr_t)q % 16) == 0 && ((uintptr_t)kv % 16) == 0 &&
             ((uintptr_t)r % 16) == 0 && ((uintptr_t)out % 16) == 0);
  if (slabs < 1 || slabs > 2 || (dv != 64 && dv != 128)) return US_ERR_UNSUPPORTED;
  CUtensorMap tmQ, tmK, tmR, tmV;
  const __nv_bfloat16* v = (const __nv_bfloat16*)kv + (long long)H * slabs * 64;
  int rc = us_tmap_2d(&tmQ, q, US_TMAP_BF16, Tq, (uint64_t)H * (slabs + 1) * 64, ldq, kBM, 64, US_SWZ_128);
  if (!rc) rc = us_tmap_2d(&tmK, kv, US_TMAP_BF16, Tk, (uint64_t)H * slabs * 64, ldkv, kBN, 64, US_SWZ_128);
  if (!rc) rc = us_tmap_2d(&tmR, r, US_TMAP_BF16, Tk, 64, 64, kBN, 64, US_SWZ_128);
  if (!rc) rc = us_tmap_2d(&tmV, v, US_TMAP_BF16, Tk, (uint64_t)H * dv, ldkv, kBN, 64, US_SWZ_128);
  if (rc) return rc;
  FlashArgs a{cu_q, cu_k, (__nv_bfloat16*)out, ldo, V, window, scale * 1.4426950408889634f, us_status_ptr(), 1,
              nullptr, 1.f, (const __nv_bfloat16*)gate, ldg, V};
  const dim3 grid((max_q + 2 * kBM - 1) / (2 * kBM), H, n_seqs);
  cudaStream_t stream = (cudaStream_t)stream_;
  if (slabs == 1) return dv == 64 ? launch_flash<1, 1, 64, 2>(tmQ, tmK, tmR, tmV, a, grid, stream)
                                  : launch_flash<1, 1, 128, 2>(tmQ, tmK, tmR, tmV, a, grid, stream);
  return dv == 64 ? launch_flash<2, 1, 64, 2>(tmQ, tmK, tmR, tmV, a, grid, stream)
                  : launch_flash<2, 1, 128, 1>(tmQ, tmK, tmR, tmV, a, grid, stream);
}

namespace {

template <bool kSig>
int grouped_flash(FlashArgs a, const void* q, long long ldq, const void* k, long long ldk, const void* v,
                  long long ldv, int n_seqs, int Tq, int Tk, int H, int G, int slabs, int dv, int max_q,
                  cudaStream_t stream) {
  US_REQUIRE(q && k && v && a.out && a.cu_q && a.cu_k && n_seqs >= 1 && Tq >= 1 && Tk >= 1 && H >= 1 && G >= 1 &&
             H % G == 0 && max_q >= 1 && a.V >= 1 && a.V <= dv);
  US_REQUIRE((ldq % 8) == 0 && (ldk % 8) == 0 && (ldv % 8) == 0 && ((uintptr_t)q % 16) == 0 &&
             ((uintptr_t)k % 16) == 0 && ((uintptr_t)v % 16) == 0 && ((uintptr_t)a.out % 16) == 0);
  if (slabs < 1 || slabs > 2 || (dv != 64 && dv != 128)) return US_ERR_UNSUPPORTED;
  CUtensorMap tmQ, tmK, tmV;
  int rc = us_tmap_2d(&tmQ, q, US_TMAP_BF16, Tq, (uint64_t)H * slabs * 64, ldq, kBM, 64, US_SWZ_128);
  if (!rc) rc = us_tmap_2d(&tmK, k, US_TMAP_BF16, Tk, (uint64_t)G * slabs * 64, ldk, kBN, 64, US_SWZ_128);
  if (!rc) rc = us_tmap_2d(&tmV, v, US_TMAP_BF16, Tk, (uint64_t)G * dv, ldv, kBN, 64, US_SWZ_128);
  if (rc) return rc;
  a.status = us_status_ptr();
  a.rep = H / G;
  const dim3 grid((max_q + 2 * kBM - 1) / (2 * kBM), H, n_seqs);
  if (slabs == 1) return dv == 64 ? launch_flash<1, 0, 64, 2, kSig>(tmQ, tmK, tmK, tmV, a, grid, stream)
                                  : launch_flash<1, 0, 128, 2, kSig>(tmQ, tmK, tmK, tmV, a, grid, stream);
  return dv == 64 ? launch_flash<2, 0, 64, 2, kSig>(tmQ, tmK, tmK, tmV, a, grid, stream)
                  : launch_flash<2, 0, 128, 2, kSig>(tmQ, tmK, tmK, tmV, a, grid, stream);
}

}  // namespace

// q [Tq, H slabs 64] rows at ldq; k [Tk, G slabs 64] and v [Tk, G dv] rows at ldk, ldv, query head h reading
// key / value head h / (H / G); V <= dv output columns per head at column h V of `out`; window 0: every
// earlier key; sink [H] or null; out_scale multiplies the output, gate [Tq, H] (rows at ldg, or null) by its
// sigmoid.  Sequences without keys are left alone.
US_API int us_window_flash(const void* q, long long ldq, const void* k, long long ldk, const void* v,
                           long long ldv, void* out, long long ldo, const int* cu_q, const int* cu_k,
                           int n_seqs, int Tq, int Tk, int H, int G, int slabs, int dv, int V, int max_q,
                           int window, float scale, const float* sink, float out_scale, const void* gate,
                           long long ldg, void* stream_) {
  FlashArgs a{cu_q, cu_k, (__nv_bfloat16*)out, ldo, V, window, scale * 1.4426950408889634f, nullptr, 1, sink,
              out_scale, (const __nv_bfloat16*)gate, ldg, 1};
  return grouped_flash<false>(a, q, ldq, k, ldk, v, ldv, n_seqs, Tq, Tk, H, G, slabs, dv, max_q,
                              (cudaStream_t)stream_);
}

// The same with weight sigmoid(cap tanh(scale temp_h (q . k) / cap) + shift_h) for a visible key (cap 0: the
// score as it is); temp and shift [H].
US_API int us_sigmoid_flash(const void* q, long long ldq, const void* k, long long ldk, const void* v,
                            long long ldv, void* out, long long ldo, const int* cu_q, const int* cu_k,
                            int n_seqs, int Tq, int Tk, int H, int G, int slabs, int dv, int V, int max_q,
                            int window, float scale, const float* temp, const float* shift, float cap,
                            float out_scale, const void* gate, long long ldg, void* stream_) {
  US_REQUIRE(temp && shift && cap >= 0.f);
  // an enormous cap: z is tiny, its tanh z itself, and cap * z the score
  FlashArgs a{cu_q, cu_k, (__nv_bfloat16*)out, ldo, V, window, 0.f, nullptr, 1, nullptr, out_scale,
              (const __nv_bfloat16*)gate, ldg, 1, temp, shift, scale, cap > 0.f ? cap : 1e9f};
  return grouped_flash<true>(a, q, ldq, k, ldk, v, ldv, n_seqs, Tq, Tk, H, G, slabs, dv, max_q,
                             (cudaStream_t)stream_);
}
