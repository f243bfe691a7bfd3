// Recurrent mixers with a delta rule, for packed batches of sequences with their state in slots of
// a pool.  The decay is a vector over the key channels of a head, or one number per head:
//
//   channel rule   S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;       o = S^T q
//   head rule      the same with a scalar g (the recurrence itself: head_delta.cu)
//   general rule   S <- diag(w) S - (a*n)(n^T S) + k v^T  (both read the old S);  o = S^T q
//
// with S [D, V] FP32 per (sequence, head).  The kernels:
//
//   us_channel_delta_prep   short causal convolutions + silu of q, k, v, unit q and k, the decay
//                           g = exp(-exp(A_log) softplus(low + dt_bias)) and beta = sigmoid(b)
//   us_head_delta_prep      the same with the decay's argument a column per head of the projection
//   us_general_delta_prep   decay w = exp(-c sigmoid(low + w0)), unit key n, removal a * n
//   us_vector_delta_rule    the recurrence
//   us_head_norm_gate       per-head RMS norm of o, weight, sigmoid or silu gate
//   us_{channel,head,general}_delta_step   all of these for one token of every sequence in one launch
//
// The preparation is parallel over tokens, so the recurrence reads finished FP32 vectors and
// does nothing but its multiply-adds.  A sequence whose first packed row stands at position 0
// starts from a zero state whatever its slot holds: slots are handed on without being cleared,
// and nothing has to be launched when a request is admitted.  A negative slot marks padding.
//
// Rule kernel: a CTA owns 32 value columns of one head of one sequence.  A lane holds D/8 rows x 2
// columns of S in registers as row pairs (packed FP32 instructions), so the two D-long reductions
// of a token are short chains and three shuffles; the read-out's is folded beside the next token's
// first one.  A token depends on the one before through one reduction and one update: that chain
// is what a long prompt costs.  The vectors of the next chunks of 8 tokens are on their way into
// a ring in shared memory meanwhile (four warps multiply, one fetches).  The state crosses HBM once per call.
#include "include/us_common.cuh"
#include "include/us_f32x2.cuh"

namespace {

using namespace us::f32x2;        // two rows of one state column per instruction

__device__ __forceinline__ float ld_any(const void* base, long long idx, int bf16) {
  return bf16 ? us::bf2f(reinterpret_cast<const __nv_bfloat16*>(base)[idx])
              : reinterpret_cast<const float*>(base)[idx];
}
__device__ __forceinline__ void st_any(void* base, long long idx, int bf16, float v) {
  if (bf16) reinterpret_cast<__nv_bfloat16*>(base)[idx] = us::f2bf(v);
  else reinterpret_cast<float*>(base)[idx] = v;
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float gate_f(float x, int silu) {
  const float s = sigmoid_f(x);
  return silu ? x * s : s;
}
__device__ __forceinline__ float softplus_f(float x) {
  return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
}

// e^x of a decay.  Hundreds of factors just below one multiply along a sequence, so a bias of
// half an ulp each would add up: near zero the rounding of 1 + (e^x - 1) is the nearest one.
__device__ __forceinline__ float decay_exp(float x) { return x > -0.5f ? 1.f + expm1f(x) : expf(x); }

// sequence that holds packed row t (cu is ascending, cu[0] = 0, cu[B] = rows)
__device__ __forceinline__ int seq_of(const int* cu, int B, int t) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

constexpr int kMaxTaps = 16;
constexpr int kMaxDim = 256;      // key channels per head
constexpr int kPrepTokens = 16;   // consecutive rows of one warp in the prefill form (<= 32)

enum Rule : int { kChannel = 0, kGeneral = 1, kHead = 2 };

struct ChannelPrep {
  const void* x;                // projection rows, element type = bf16 flag
  long long ldx;
  int off_q, off_k, off_v, off_b;
  const float *cq, *ck, *cv;    // taps [channels, K]
  const float* low;             // [rows, H * D], or null: a decay per head from column off_a
  long long ldlow;
  int off_a;
  const float *A_log, *dt_bias; // [H], [H * D] (per head: [H])
  void* conv;                   // [slots, K, C], C = 2 Hk D + H V: input of position p in entry p % K
  float *q, *k, *v, *g, *beta;  // [rows, Hk, D] x 2, [rows, H, V], [rows, H, D] or [rows, H], [rows, H]
  const int *cu, *slots, *pos;
  int B, rows, H, Hk, D, V, K, bf16, one_token;
};

// The last inputs of a sequence's convolutions are a ring of K entries addressed by position:
// a token reads K - 1 entries and writes another one, so nothing is shifted and the readers of
// one token never meet its writer.  Positions before the sequence are zero.

// A warp owns one head of q, of k, of v or of the decay for kPrepTokens consecutive rows (prefill)
// or one row (every sequence brings one token: the warp then also stores its channels' inputs).
// The window of a channel stays in registers from row to row (KT >= K taps, leading ones zero).
// NI: channels per lane.
template <int KT, int NI>
__global__ void __launch_bounds__(256) channel_prep_kernel(const ChannelPrep a) {
  US_PDL_PROLOGUE();
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.y * 8 + (threadIdx.x >> 5);
  const int units = 2 * a.Hk + 2 * a.H;
  if (unit >= units) return;
  const int per = a.one_token ? 1 : kPrepTokens;
  const int t0 = blockIdx.x * per, t1 = min(a.rows, t0 + per);
  if (unit >= 2 * a.Hk + a.H) {                       // decay and step size
    const int h = unit - 2 * a.Hk - a.H;
    const float A = expf(a.A_log[h]);
    if (!a.low) {                                     // a lane per row
      if (t0 + lane < t1) {
        const long long row = t0 + lane, at = row * a.H + h;
        a.g[at] = decay_exp(-A * softplus_f(ld_any(a.x, row * a.ldx + a.off_a + h, a.bf16) + a.dt_bias[h]));
        a.beta[at] = sigmoid_f(ld_any(a.x, row * a.ldx + a.off_b + h, a.bf16));
      }
      return;
    }
#pragma unroll 2
    for (int t = t0; t < t1; ++t) {
      const float* lo = a.low + (long long)t * a.ldlow + (long long)h * a.D;
      float* g = a.g + ((long long)t * a.H + h) * a.D;
      for (int d = lane; d < a.D; d += 32)
        g[d] = decay_exp(-A * softplus_f(lo[d] + a.dt_bias[h * a.D + d]));
      if (lane == 0)
        a.beta[(long long)t * a.H + h] =
            sigmoid_f(ld_any(a.x, (long long)t * a.ldx + a.off_b + h, a.bf16));
    }
    return;
  }
  int head, dim, off, cbase;
  const float* taps;
  if (unit < a.Hk) {
    head = unit; dim = a.D; off = a.off_q + head * a.D; taps = a.cq + (long long)head * a.D * a.K;
    cbase = head * a.D;
  } else if (unit < 2 * a.Hk) {
    head = unit - a.Hk; dim = a.D; off = a.off_k + head * a.D;
    taps = a.ck + (long long)head * a.D * a.K;
    cbase = a.Hk * a.D + head * a.D;
  } else {
    head = unit - 2 * a.Hk; dim = a.V; off = a.off_v + head * a.V;
    taps = a.cv + (long long)head * a.V * a.K;
    cbase = 2 * a.Hk * a.D + head * a.V;
  }
  const long long C = 2LL * a.Hk * a.D + (long long)a.H * a.V;
  float w[NI][KT], win[NI][KT];                       // win[KT - 1]: the current row
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int j = 0; j < KT; ++j) {
      const int d = i * 32 + lane, c = j - (KT - a.K);
      w[i][j] = (c >= 0 && d < dim) ? taps[(long long)d * a.K + c] : 0.f;
    }
  int s = seq_of(a.cu, a.B, t0), end = t0, slot = -1;
  for (int t = t0; t < t1; ++t) {
    if (t >= end) {                                   // first row here, or of the next sequence
      while (a.cu[s + 1] <= t) ++s;
      const int start = a.cu[s], p0 = a.pos[start];
      end = a.cu[s + 1];
      slot = a.slots[s];
      const long long sbase = (long long)max(slot, 0) * a.K * C + cbase;
#pragma unroll
      for (int j = 1; j < KT; ++j) {                  // entry of the row KT - j back, before t
        const int src = t - (KT - j), pos = p0 + src - start;
        const bool in_x = src >= start, in_ring = !in_x && pos >= 0 && KT - j < a.K && slot >= 0;
        const long long at = in_ring ? sbase + (long long)(pos % a.K) * C : 0;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          const int d = i * 32 + lane;
          float v = 0.f;
          if (d < dim) {
            if (in_x) v = ld_any(a.x, (long long)src * a.ldx + off + d, a.bf16);
            else if (in_ring) v = ld_any(a.conv, at + d, a.bf16);
          }
          win[i][j] = v;
        }
      }
      if (a.one_token && a.K > 1 && slot >= 0) {
        const long long at1 = sbase + (long long)(p0 % a.K) * C;
#pragma unroll
        for (int i = 0; i < NI; ++i)
          if (i * 32 + lane < dim)
            st_any(a.conv, at1 + i * 32 + lane, a.bf16,
                   ld_any(a.x, (long long)t * a.ldx + off + i * 32 + lane, a.bf16));
      }
    }
    // the window moves on: entries 1 .. KT - 1 become the older ones of this row
    float y[NI], ss = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = i * 32 + lane;
#pragma unroll
      for (int j = 0; j + 1 < KT; ++j) win[i][j] = win[i][j + 1];
      win[i][KT - 1] = d < dim ? ld_any(a.x, (long long)t * a.ldx + off + d, a.bf16) : 0.f;
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < KT; ++j) acc = fmaf(w[i][j], win[i][j], acc);
      y[i] = acc / (1.f + expf(-acc));
      ss += y[i] * y[i];
    }
    if (slot < 0) continue;
    if (unit < 2 * a.Hk) {
      float inv = 1.f / sqrtf(us::warp_sum(ss) + 1e-6f);
      if (unit < a.Hk) inv *= 1.f / sqrtf((float)a.D);
      float* dst = (unit < a.Hk ? a.q : a.k) + ((long long)t * a.Hk + head) * a.D;
#pragma unroll
      for (int i = 0; i < NI; ++i)
        if (i * 32 + lane < dim) dst[i * 32 + lane] = y[i] * inv;
    } else {
      float* dst = a.v + ((long long)t * a.H + head) * a.V;
#pragma unroll
      for (int i = 0; i < NI; ++i)
        if (i * 32 + lane < dim) dst[i * 32 + lane] = y[i];
    }
  }
}

// Inputs of every sequence's last K - 1 rows into its ring, after the rows' convolutions.
__global__ void __launch_bounds__(256) conv_ring_kernel(const ChannelPrep a) {
  US_PDL_PROLOGUE();
  const int c = blockIdx.x * 256 + threadIdx.x;
  const int nq = a.Hk * a.D, C = 2 * nq + a.H * a.V;
  if (c >= C) return;
  const int s = blockIdx.y;
  const int start = a.cu[s], T = a.cu[s + 1] - start, slot = a.slots[s];
  if (slot < 0 || T <= 0) return;
  const int p0 = a.pos[start];
  const int col = c < nq ? a.off_q + c : c < 2 * nq ? a.off_k + c - nq : a.off_v + c - 2 * nq;
  for (int t = max(0, T - (a.K - 1)); t < T; ++t)
    st_any(a.conv, ((long long)slot * a.K + (p0 + t) % a.K) * C + c, a.bf16,
           ld_any(a.x, (long long)(start + t) * a.ldx + col, a.bf16));
}

struct GeneralPrep {
  const void* x;
  long long ldx;
  int off_r, off_k, off_v, off_a;
  const float* low;             // [rows, H * D] (before w0)
  long long ldlow;
  const float *w0, *a_bias;     // [H * D]
  float *w, *n, *p, *k, *r, *v;  // [rows, H, D]
  int rows, H, D, bf16;
  float rate;                   // w = exp(-rate * sigmoid(.))
};

// One warp per (row, head).
__global__ void __launch_bounds__(256) general_prep_kernel(const GeneralPrep a) {
  US_PDL_PROLOGUE();
  const long long r = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (r >= (long long)a.rows * a.H) return;
  const int t = (int)(r / a.H), h = (int)(r - (long long)t * a.H);
  const long long xr = (long long)t * a.ldx + (long long)h * a.D;
  float kv[kMaxDim / 32], ss = 0.f;
#pragma unroll
  for (int i = 0; i < kMaxDim / 32; ++i) {
    const int d = i * 32 + lane;
    kv[i] = d < a.D ? ld_any(a.x, xr + a.off_k + d, a.bf16) : 0.f;
    ss += kv[i] * kv[i];
  }
  const float inv = 1.f / sqrtf(us::warp_sum(ss) + 1e-6f);
#pragma unroll
  for (int i = 0; i < kMaxDim / 32; ++i) {
    const int d = i * 32 + lane;
    if (d >= a.D) continue;
    const int hd = h * a.D + d;
    const float n = kv[i] * inv;
    a.k[r * a.D + d] = kv[i];
    a.r[r * a.D + d] = ld_any(a.x, xr + a.off_r + d, a.bf16);
    a.v[r * a.D + d] = ld_any(a.x, xr + a.off_v + d, a.bf16);
    a.w[r * a.D + d] =
        decay_exp(-a.rate * sigmoid_f(a.low[(long long)t * a.ldlow + hd] + a.w0[hd]));
    a.n[r * a.D + d] = n;
    a.p[r * a.D + d] = n * sigmoid_f(ld_any(a.x, xr + a.off_a + d, a.bf16) + a.a_bias[hd]);
  }
}

constexpr int kCols = 32;         // value columns per CTA
constexpr int kRuleCompute = 128, kRuleCopy = 32;    // threads that multiply / that fetch vectors
constexpr int kRuleThreads = kRuleCompute + kRuleCopy;
constexpr int kRuleBufs = 4;                         // chunks of vectors in shared memory

struct RuleArgs {
  const float *q, *k, *v;         // [rows, Hk, D] x 2, [rows, H, V]
  const float* g;                 // decay [rows, H, D]
  const float* n;                 // general: removal direction [rows, H, D]
  const float* p;                 // general: removal rate * direction [rows, H, D]
  const float* beta;              // channel: [rows, H]
  float* state;                   // [slots, H, D, V]
  float* out;                     // [rows, H, V]
  const int *cu, *slots, *pos;
  int H, Hk, D, V;
};

// Folds two per-lane column sums over the 8 lanes that span the rows: afterwards lanes 0 .. 3 hold
// column 0's sum, lanes 4 .. 7 column 1's.
__device__ __forceinline__ float fold8(float c0, float c1, bool up) {
  float s = (up ? c1 : c0) + __shfl_xor_sync(0xffffffffu, up ? c0 : c1, 4);
  s += __shfl_xor_sync(0xffffffffu, s, 2);
  s += __shfl_xor_sync(0xffffffffu, s, 1);
  return s;
}

template <int BYTES>
__device__ __forceinline__ void cp_async(float* dst, const float* src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  if (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

// A token in shared memory: kVecs vectors of DP floats (g, k, q and, general, n, p), then 32
// columns of v and beta.
template <int DP, bool GENERAL>
struct Stage {
  static constexpr int kVecs = GENERAL ? 5 : 3;
  static constexpr int kToken = kVecs * DP + kCols + 4;
  static constexpr int kChunk = 8;                    // tokens per chunk
  static constexpr int kFloats = kChunk * kToken;
};

// Asynchronous copies of tokens' vectors by the copying threads.  Widths that are multiples of
// four move as 16-byte pieces: a thread owns the same pieces of every token and only advances its
// pointers (address arithmetic per piece would cost as much as the recurrence).
template <int DP, bool GENERAL>
struct Copier {
  using St = Stage<DP, GENERAL>;
  static constexpr int kQ = DP / 4;
  static constexpr int kPieces = St::kVecs * kQ + kCols / 4;
  static constexpr int kMine = (kPieces + kRuleCopy - 1) / kRuleCopy;
  const float* src[kMine];
  int step[kMine], dst[kMine];          // floats per token, place in the token (-1: nothing)
  const float* beta;
  int tid, heads;
  bool quad;
  __device__ __forceinline__ void init(const RuleArgs& a, int tid_, long long row0, int h, int hk, int col0) {
    tid = tid_;
    heads = a.H;
    quad = (a.V & 3) == 0 && (a.D & 3) == 0;
    beta = GENERAL ? nullptr : a.beta + row0 * a.H + h;
#pragma unroll
    for (int i = 0; i < kMine; ++i) {
      const int e = tid + i * kRuleCopy, vec = e / kQ, d = (e - vec * kQ) * 4;
      dst[i] = -1;
      src[i] = nullptr;
      step[i] = 0;
      if (e < St::kVecs * kQ) {
        if (d >= a.D) continue;
        const bool shared = vec == 1 || vec == 2;
        const int heads_ = shared ? a.Hk : a.H, hh = shared ? hk : h;
        src[i] = (vec == 1 ? a.k : vec == 2 ? a.q : vec == 0 ? a.g : vec == 3 ? a.n : a.p) +
                 (row0 * heads_ + hh) * a.D + d;
        step[i] = heads_ * a.D;
        dst[i] = vec * DP + d;
      } else if (e < kPieces) {
        const int c = (e - St::kVecs * kQ) * 4;
        if (col0 + c >= a.V) continue;
        src[i] = a.v + (row0 * a.H + h) * a.V + col0 + c;
        step[i] = a.H * a.V;
        dst[i] = St::kVecs * DP + c;
      }
    }
  }
  // the next n tokens into buf (row0: their first row, for widths that are not multiples of 4)
  __device__ __forceinline__ void fetch(const RuleArgs& a, float* buf, int n, long long row0, int h, int hk,
                                        int col0) {
    if (quad) {
      for (int t = 0; t < n; ++t, buf += St::kToken) {
#pragma unroll
        for (int i = 0; i < kMine; ++i)
          if (dst[i] >= 0) {
            cp_async<16>(buf + dst[i], src[i]);
            src[i] += step[i];
          }
        if (!GENERAL && tid == 0) {
          cp_async<4>(buf + St::kVecs * DP + kCols, beta);
          beta += heads;
        }
      }
    } else {
      for (int t = 0; t < n; ++t, buf += St::kToken) {
        const long long row = row0 + t;
        for (int e = tid; e < St::kVecs * a.D; e += kRuleCopy) {
          const int vec = e / a.D, d = e - vec * a.D;
          const bool shared = vec == 1 || vec == 2;
          const float* from = vec == 1 ? a.k : vec == 2 ? a.q : vec == 0 ? a.g : vec == 3 ? a.n : a.p;
          cp_async<4>(buf + vec * DP + d, from + (shared ? row * a.Hk + hk : row * a.H + h) * a.D + d);
        }
        for (int c = tid; c < kCols && col0 + c < a.V; c += kRuleCopy)
          cp_async<4>(buf + St::kVecs * DP + c, a.v + (row * a.H + h) * a.V + col0 + c);
        if (!GENERAL && tid == 0) cp_async<4>(buf + St::kVecs * DP + kCols, a.beta + row * a.H + h);
      }
    }
  }
};

template <int DP, bool GENERAL>
__global__ void __launch_bounds__(kRuleThreads, DP > 128 ? 1 : 3) vector_delta_kernel(const RuleArgs a) {
  US_PDL_PROLOGUE();
  using St = Stage<DP, GENERAL>;
  constexpr int NG = DP / 32;                         // groups of four rows per lane
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, s = blockIdx.z;
  const int hk = h / (a.H / a.Hk);
  const int col0 = blockIdx.x * kCols;
  const int start = a.cu[s], T = a.cu[s + 1] - start, slot = a.slots[s];
  if (T <= 0) return;
  if (slot < 0) {                                     // padding: defined rows, no state
    for (int e = tid; e < T * kCols; e += kRuleThreads) {
      const int t = e / kCols, c = col0 + e - t * kCols;
      if (c < a.V) a.out[((long long)(start + t) * a.H + h) * a.V + c] = 0.f;
    }
    return;
  }
  const bool gaps = a.D < DP || col0 + kCols > a.V;    // places that no copy fills: zero
  if (gaps) {
    for (int e = tid; e < kRuleBufs * St::kFloats; e += kRuleThreads) sm[e] = 0.f;
    __syncthreads();
  }
  if (tid >= kRuleCompute) {                          // the copying threads stay one chunk ahead
    Copier<DP, GENERAL> cp;
    cp.init(a, tid - kRuleCompute, start, h, hk, col0);
    const int chunks = (T + St::kChunk - 1) / St::kChunk;
    auto fetch = [&](int r) {                         // (an empty group past the end)
      if (r < chunks)
        cp.fetch(a, sm + (r % kRuleBufs) * St::kFloats, min(St::kChunk, T - r * St::kChunk),
                 start + r * St::kChunk, h, hk, col0);
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll 1
    for (int r = 0; r < kRuleBufs - 1; ++r) fetch(r);
#pragma unroll 1
    for (int r = 0; r < chunks; ++r) {
      asm volatile("cp.async.wait_group %0;" ::"n"(kRuleBufs - 2) : "memory");
      __syncthreads();                                // chunk r is there, chunk r - 1 consumed
      fetch(r + kRuleBufs - 1);
    }
    return;
  }
  const int kq = lane & 7;                                         // lane's share of the rows
  const bool up = kq >= 4;                                         // a fold leaves column 1 here
  const int cb = warp * 8 + (lane >> 3) * 2;                       // the lane's two columns
  float* Sg = a.state + (((long long)slot * a.H + h) * a.D) * a.V + col0 + cb;
  const bool wide = (a.V & 1) == 0;
  const bool fresh = a.pos[start] == 0;
  const bool c0ok = col0 + cb < a.V, c1ok = col0 + cb + 1 < a.V;
  f2 S[NG * 2][2];                                    // row pairs x 2 columns
#pragma unroll
  for (int j = 0; j < NG; ++j)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float2 x[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int row = (j * 8 + kq) * 4 + e * 2 + i;
        x[i] = make_float2(0.f, 0.f);
        if (!fresh && row < a.D) {
          const float* p = Sg + (long long)row * a.V;
          if (wide && c0ok) {
            x[i] = *reinterpret_cast<const float2*>(p);
          } else {
            if (c0ok) x[i].x = p[0];
            if (c1ok) x[i].y = p[1];
          }
        }
      }
      S[j * 2 + e][0] = pack2(x[0].x, x[1].x);
      S[j * 2 + e][1] = pack2(x[0].y, x[1].y);
    }
  float* op = a.out + ((long long)start * a.H + h) * a.V + col0 + cb + (up ? 1 : 0);
  const bool writes = (lane & 3) == 0 && (up ? c1ok : c0ok);
  const long long ostep = (long long)a.H * a.V;
  // the read-out of a token is folded beside the next token's first reduction: two independent
  // shuffle chains instead of one after the other
  float o0 = 0.f, o1 = 0.f;
  bool pending = false;
  int buf = 0;
  for (int c0 = 0; c0 < T; c0 += St::kChunk, buf = buf + 1 == kRuleBufs ? 0 : buf + 1) {
    const int n = min(St::kChunk, T - c0);
    __syncthreads();                                  // this chunk's vectors are there
    const float* base = sm + buf * St::kFloats;
    for (int t = 0; t < n; ++t, base += St::kToken) {
      const float* vs = base + St::kVecs * DP;
      f2 y[2][2] = {{0ull, 0ull}, {0ull, 0ull}};
#pragma unroll
      for (int j = 0; j < NG; ++j) {
        const int r0 = (j * 8 + kq) * 4;
        f2 m[2];
        if (GENERAL) {
          lds_vec(m, base + 3 * DP + r0);
        } else {
          f2 g[2];
          lds_vec(m, base + DP + r0);
          lds_vec(g, base + r0);
#pragma unroll
          for (int e = 0; e < 2; ++e)
#pragma unroll
            for (int c = 0; c < 2; ++c)     // the key sees the decayed state
              S[j * 2 + e][c] = mul2(S[j * 2 + e][c], g[e]);
        }
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int c = 0; c < 2; ++c) y[c][e] = fma2(S[j * 2 + e][c], m[e], y[c][e]);
      }
      y[0][0] = add2(y[0][0], y[0][1]);
      y[1][0] = add2(y[1][0], y[1][1]);
      const float seen = fold8(lo2(y[0][0]) + hi2(y[0][0]), lo2(y[1][0]) + hi2(y[1][0]), up);
      const float o = fold8(o0, o1, up);
      if (pending) {
        if (writes) *op = o;
        op += ostep;
      }
      pending = true;
      float c = seen;                               // general: n^T S of this lane's column
      if (!GENERAL) c = vs[kCols] * (vs[cb + (up ? 1 : 0)] - seen);
      const float other = __shfl_xor_sync(0xffffffffu, c, 4);
      const float u0 = up ? other : c, u1 = up ? c : other;
      f2 uu[2], vv[2];
      if (GENERAL) {
        const float2 v2 = *reinterpret_cast<const float2*>(vs + cb);
        uu[0] = pack2(-u0, -u0); uu[1] = pack2(-u1, -u1);
        vv[0] = pack2(v2.x, v2.x); vv[1] = pack2(v2.y, v2.y);
      } else {
        uu[0] = pack2(u0, u0); uu[1] = pack2(u1, u1);
      }
      f2 oo[2][2] = {{0ull, 0ull}, {0ull, 0ull}};
#pragma unroll
      for (int j = 0; j < NG; ++j) {
        const int r0 = (j * 8 + kq) * 4;
        f2 k[2], q[2], g[2], p[2];
        lds_vec(k, base + DP + r0);
        lds_vec(q, base + 2 * DP + r0);
        if (GENERAL) {
          lds_vec(g, base + r0);
          lds_vec(p, base + 4 * DP + r0);
        }
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            f2& x = S[j * 2 + e][c];
            if (GENERAL) x = fma2(k[e], vv[c], fma2(p[e], uu[c], mul2(g[e], x)));
            else x = fma2(k[e], uu[c], x);
            oo[c][e] = fma2(x, q[e], oo[c][e]);
          }
      }
      oo[0][0] = add2(oo[0][0], oo[0][1]);
      oo[1][0] = add2(oo[1][0], oo[1][1]);
      o0 = lo2(oo[0][0]) + hi2(oo[0][0]);
      o1 = lo2(oo[1][0]) + hi2(oo[1][0]);
    }
  }
  const float o = fold8(o0, o1, up);
  if (writes) *op = o;
#pragma unroll
  for (int j = 0; j < NG; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int row = (j * 8 + kq) * 4 + e;
      if (row >= a.D) continue;
      float* p = Sg + (long long)row * a.V;
      const f2 s0 = S[j * 2 + e / 2][0], s1 = S[j * 2 + e / 2][1];
      const float x0 = (e & 1) ? hi2(s0) : lo2(s0), x1 = (e & 1) ? hi2(s1) : lo2(s1);
      if (wide && c0ok) {
        *reinterpret_cast<float2*>(p) = make_float2(x0, x1);
      } else {
        if (c0ok) p[0] = x0;
        if (c1ok) p[1] = x1;
      }
    }
}

// y = o / rms(o over V) * w * sigmoid(gate) (or silu), one warp per (row, head); columns past H * V of
// the (padded) output row are zeroed by the last head's warp.
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ w, int w_head_stride,
                      const void* __restrict__ gate, long long ldg, void* __restrict__ y,
                      long long ldy, int rows, int H, int V, float eps, int bf16, int gate_bf16,
                      int silu) {
  US_PDL_PROLOGUE();
  const long long r = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (r >= (long long)rows * H) return;
  const int t = (int)(r / H), h = (int)(r - (long long)t * H);
  const float* x = o + r * V;
  float ss = 0.f;
  for (int c = lane; c < V; c += 32) ss += x[c] * x[c];
  const float inv = 1.f / sqrtf(us::warp_sum(ss) / (float)V + eps);
  for (int c = lane; c < V; c += 32) {
    const float gv = ld_any(gate, (long long)t * ldg + h * V + c, gate_bf16);
    st_any(y, (long long)t * ldy + h * V + c, bf16,
           x[c] * inv * w[h * w_head_stride + c] * gate_f(gv, silu));
  }
  if (h == H - 1)
    for (long long c = (long long)H * V + lane; c < ldy; c += 32)
      st_any(y, (long long)t * ldy + c, bf16, 0.f);
}

// ------------------------------------------------------------- decode step --
struct StepArgs {
  const void* x;                  // projection rows
  long long ldx;
  int off_q, off_k, off_v, off_b; // general: read-out, key, value, removal rate
  const float *cq, *ck, *cv;      // channel: taps
  const float* low;               // [B, H * D]
  long long ldlow;
  int off_a;                      // head: column of the decay's argument
  const float *A_log, *bias;      // channel: [H], dt_bias [H * D]; head: [H] x 2; general: null, w0 [H * D]
  const float* a_bias;            // general: [H * D]
  void* conv;                     // channel: ring [slots, K, C]
  float* state;                   // [slots, H, D, V]
  const float* nw;                // norm weight
  int nw_head_stride;
  const void* gate;               // [B, H * V] at ldg
  long long ldg;
  void* y;                        // [B, ldy]
  long long ldy;
  const int *slots, *pos;
  int H, Hk, D, V, K, bf16, gate_bf16, silu;
  float eps, rate;
};

constexpr int kStepThreads = 256;

// One token of every sequence through a whole mixer between its input and output projections:
// convolutions (channel) or key norm (general), decay, recurrence, per-head norm and gate.  A CTA
// owns one head of one sequence.  A thread holds R rows x 4 columns of S, a warp reading whole
// rows; the state is on its way while the vectors are formed in shared memory.  LQ threads span
// the value columns.  Sums over key channels meet in shared memory.
template <int R, int LQ, int RULE>
__global__ void __launch_bounds__(kStepThreads) vector_delta_step_kernel(const StepArgs a) {
  US_PDL_PROLOGUE();
  constexpr bool GENERAL = RULE == kGeneral;
  constexpr int kVecs = RULE == kHead ? 2 : 3;        // vectors of D formed before v
  constexpr int RG = kStepThreads / LQ;               // row groups
  __shared__ float qs[kMaxDim], ks[kMaxDim], gs[RULE == kHead ? 1 : kMaxDim], ps[GENERAL ? kMaxDim : 1],
      vs[LQ * 4];
  __shared__ __align__(16) float red[RG][LQ * 4];
  __shared__ float scal[5];                           // 1 / |q|, 1 / |k|, beta, (norm's second part), decay
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int slot = a.slots[b], H = a.H, D = a.D, V = a.V;
  if (slot < 0) {
    for (int c = tid; c < V; c += kStepThreads) st_any(a.y, b * a.ldy + h * V + c, a.bf16, 0.f);
    return;
  }
  const int p0 = a.pos[b], cq4 = (tid % LQ) * 4, rg = tid / LQ;
  const bool on = cq4 < V;
  float* Sg = a.state + ((long long)slot * H + h) * D * V + cq4;
  float4 S[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int row = rg + i * RG;
    S[i] = (p0 > 0 && on && row < D) ? *reinterpret_cast<const float4*>(Sg + (long long)row * V)
                                     : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const long long xb = b * a.ldx;
  const int hk = h / (H / a.Hk);
  // ---- vectors ----
  for (int e = tid; e < kVecs * D + V; e += kStepThreads) {
    const int what = e < D ? 0 : e < 2 * D ? 1 : e < kVecs * D ? 2 : 3;   // q, k, decay, v
    const int d = e - (what == 3 ? kVecs : what) * D;
    if (RULE != kHead && what == 2) {
      const float lo = a.low[b * a.ldlow + h * D + d] + a.bias[h * D + d];
      if (GENERAL) {
        gs[d] = decay_exp(-a.rate * sigmoid_f(lo));
        ps[d] = sigmoid_f(ld_any(a.x, xb + a.off_b + h * D + d, a.bf16) + a.a_bias[h * D + d]);
      } else {
        gs[d] = decay_exp(-expf(a.A_log[h]) * softplus_f(lo));
      }
      continue;
    }
    float v;
    if (GENERAL) {
      const int off = what == 0 ? a.off_q : what == 1 ? a.off_k : a.off_v;
      v = ld_any(a.x, xb + off + h * (what == 3 ? V : D) + d, a.bf16);
    } else {
      const int nq = a.Hk * D, C = 2 * nq + H * V;
      const int ch = what == 3 ? h * V + d : hk * D + d;                  // channel of q, k or v
      const int col = (what == 0 ? a.off_q : what == 1 ? a.off_k : a.off_v) + ch;
      const float* taps = (what == 0 ? a.cq : what == 1 ? a.ck : a.cv) + (long long)ch * a.K;
      const long long ring = (long long)slot * a.K * C + (what == 3 ? 2 * nq : what == 1 ? nq : 0) + ch;
      const float cur = ld_any(a.x, xb + col, a.bf16);
      float acc = taps[a.K - 1] * cur;
#pragma unroll
      for (int j = 1; j < kMaxTaps; ++j)
        if (j < a.K && p0 - j >= 0)
          acc += taps[a.K - 1 - j] * ld_any(a.conv, ring + (long long)((p0 - j) % a.K) * C, a.bf16);
      // the entry written is one that no reader of this token touches
      if (a.K > 1 && (what == 3 || h % (H / a.Hk) == 0))
        st_any(a.conv, ring + (long long)(p0 % a.K) * C, a.bf16, cur);
      v = acc / (1.f + expf(-acc));
    }
    (what == 0 ? qs : what == 1 ? ks : vs)[d] = v;
  }
  __syncthreads();
  if (warp < 2) {                                      // unit lengths of q and k
    const float* x = warp ? ks : qs;
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) ss += x[d] * x[d];
    ss = us::warp_sum(ss);
    if (lane == 0) scal[warp] = 1.f / sqrtf(ss + 1e-6f);
  } else if (!GENERAL && tid == 64) {
    scal[2] = sigmoid_f(ld_any(a.x, xb + a.off_b + h, a.bf16));
    if (RULE == kHead)
      scal[4] = decay_exp(-expf(a.A_log[h]) * softplus_f(ld_any(a.x, xb + a.off_a + h, a.bf16) + a.bias[h]));
  }
  __syncthreads();
  const float kinv = scal[1];
  // ---- what the key sees ----
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int row = rg + i * RG;
    if (row >= D) break;
    const float k = ks[row] * kinv;
    if (!GENERAL) {
      const float g = RULE == kHead ? scal[4] : gs[row];
      S[i].x *= g; S[i].y *= g; S[i].z *= g; S[i].w *= g;
    }
    acc.x = fmaf(S[i].x, k, acc.x); acc.y = fmaf(S[i].y, k, acc.y);
    acc.z = fmaf(S[i].z, k, acc.z); acc.w = fmaf(S[i].w, k, acc.w);
  }
  auto gather = [&](float4 x) {                        // sum over the row groups
    *reinterpret_cast<float4*>(&red[rg][cq4]) = x;
    __syncthreads();
    float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < RG; ++r) {
      const float4 e = *reinterpret_cast<const float4*>(&red[r][cq4]);
      t.x += e.x; t.y += e.y; t.z += e.z; t.w += e.w;
    }
    return t;
  };
  const float4 seen = gather(acc);
  float4 vv = make_float4(0.f, 0.f, 0.f, 0.f), u = seen;
  if (on) vv = make_float4(vs[cq4], vs[cq4 + 1], vs[cq4 + 2], vs[cq4 + 3]);
  if (!GENERAL) {
    const float beta = scal[2];
    u = make_float4(beta * (vv.x - seen.x), beta * (vv.y - seen.y), beta * (vv.z - seen.z),
                    beta * (vv.w - seen.w));
  }
  acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int row = rg + i * RG;
    if (row >= D) break;
    float4& x = S[i];
    if (GENERAL) {
      const float g = gs[row], k = ks[row], p = ps[row] * (k * kinv);
      x.x = fmaf(k, vv.x, fmaf(-p, u.x, g * x.x)); x.y = fmaf(k, vv.y, fmaf(-p, u.y, g * x.y));
      x.z = fmaf(k, vv.z, fmaf(-p, u.z, g * x.z)); x.w = fmaf(k, vv.w, fmaf(-p, u.w, g * x.w));
    } else {
      const float k = ks[row] * kinv;
      x.x = fmaf(k, u.x, x.x); x.y = fmaf(k, u.y, x.y);
      x.z = fmaf(k, u.z, x.z); x.w = fmaf(k, u.w, x.w);
    }
    const float q = qs[row];
    acc.x = fmaf(x.x, q, acc.x); acc.y = fmaf(x.y, q, acc.y);
    acc.z = fmaf(x.z, q, acc.z); acc.w = fmaf(x.w, q, acc.w);
    if (on) *reinterpret_cast<float4*>(Sg + (long long)row * V) = x;
  }
  __syncthreads();                                     // the first sum has been read
  float4 o = gather(acc);
  const float qscale = GENERAL ? 1.f : scal[0] / sqrtf((float)D);
  o.x *= qscale; o.y *= qscale; o.z *= qscale; o.w *= qscale;
  // ---- norm over the head's values, weight, gate ----
  if (warp >= (LQ + 31) / 32) return;                  // the first LQ threads hold the head once
  float ss = (tid < LQ && on) ? o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w : 0.f;
  ss = us::warp_sum(ss);
  if (LQ > 32) {
    if (lane == 0) scal[2 + warp] = ss;                // (beta has been read)
    asm volatile("bar.sync 1, 64;" ::: "memory");
    ss = scal[2] + scal[3];
  }
  if (tid >= LQ || !on) return;
  const float inv = 1.f / sqrtf(ss / (float)V + a.eps);
  const float r[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int c = h * V + cq4 + i;
    st_any(a.y, b * a.ldy + c, a.bf16,
           r[i] * inv * a.nw[h * a.nw_head_stride + cq4 + i] * gate_f(ld_any(a.gate, b * a.ldg + c, a.gate_bf16), a.silu));
  }
}

template <int LQ, int RULE>
int launch_step(const StepArgs& a, int B, cudaStream_t stream) {
  const int rows = (a.D + kStepThreads / LQ - 1) / (kStepThreads / LQ);
  const dim3 grid(a.H, B), block(kStepThreads);
  if (rows <= 4) US_CUDA_CHECK(us::launch_pdl(vector_delta_step_kernel<4, LQ, RULE>, grid, block, 0, stream, a));
  else if (rows <= 8) US_CUDA_CHECK(us::launch_pdl(vector_delta_step_kernel<8, LQ, RULE>, grid, block, 0, stream, a));
  else if (rows <= 16) US_CUDA_CHECK(us::launch_pdl(vector_delta_step_kernel<16, LQ, RULE>, grid, block, 0, stream, a));
  else return US_ERR_UNSUPPORTED;
  return US_OK;
}

template <int RULE>
int step_impl(const StepArgs& a, int B, cudaStream_t stream) {
  US_REQUIRE(a.x && (a.low || RULE == kHead) && a.bias && a.state && a.nw && a.gate && a.y && a.slots && a.pos && B >= 1 &&
             B <= 65535 && a.H >= 1 && a.ldy == (long long)a.H * a.V && ((uintptr_t)a.state % 16) == 0);
  if (a.D < 1 || a.D > kMaxDim || (a.V & 3) || a.V > 256) return US_ERR_UNSUPPORTED;
  if (a.V <= 64) return launch_step<16, RULE>(a, B, stream);
  if (a.V <= 128) return launch_step<32, RULE>(a, B, stream);
  return launch_step<64, RULE>(a, B, stream);
}

template <int DP, bool GENERAL>
int launch_rule(const RuleArgs& a, int B, cudaStream_t stream) {
  constexpr size_t smem = kRuleBufs * Stage<DP, GENERAL>::kFloats * sizeof(float);
  static bool configured = false;
  if (!configured && smem > 48 * 1024) {
    US_CUDA_CHECK(cudaFuncSetAttribute(vector_delta_kernel<DP, GENERAL>,
                                       cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  }
  configured = true;
  US_CUDA_CHECK(us::launch_pdl(vector_delta_kernel<DP, GENERAL>,
                               dim3((a.V + kCols - 1) / kCols, a.H, B), dim3(kRuleThreads), smem,
                               stream, a));
  return US_OK;
}

int prep_impl(const ChannelPrep& a, cudaStream_t stream) {
  US_REQUIRE(a.x && a.cq && a.ck && a.cv && a.A_log && a.dt_bias && a.q && a.k && a.v && a.g && a.beta && a.cu &&
             a.slots && a.pos && a.B >= 1 && a.rows >= 1 && a.H >= 1 && a.Hk >= 1 && a.H % a.Hk == 0);
  US_REQUIRE(a.K == 1 || a.conv);
  US_REQUIRE(!a.one_token || a.rows == a.B);
  if (a.K < 1 || a.K > kMaxTaps || a.D < 1 || a.D > kMaxDim || a.V < 1 || a.V > kMaxDim)
    return US_ERR_UNSUPPORTED;
  const int per = a.one_token ? 1 : kPrepTokens;
  const int units = 2 * a.Hk + 2 * a.H;
  const dim3 grid((a.rows + per - 1) / per, (units + 7) / 8);
  const int widest = a.D > a.V ? a.D : a.V;
#define US_PREP(KT)                                                                               \
  if (widest <= 64) US_CUDA_CHECK(us::launch_pdl(channel_prep_kernel<KT, 2>, grid, dim3(256), 0, stream, a));       \
  else if (widest <= 128) US_CUDA_CHECK(us::launch_pdl(channel_prep_kernel<KT, 4>, grid, dim3(256), 0, stream, a)); \
  else US_CUDA_CHECK(us::launch_pdl(channel_prep_kernel<KT, 8>, grid, dim3(256), 0, stream, a));
  if (a.K <= 4) { US_PREP(4) } else if (a.K <= 8) { US_PREP(8) } else { US_PREP(16) }
#undef US_PREP
  if (!a.one_token && a.K > 1)
    US_CUDA_CHECK(us::launch_pdl(conv_ring_kernel, dim3((2 * a.Hk * a.D + a.H * a.V + 255) / 256, a.B),
                                 dim3(256), 0, stream, a));
  return US_OK;
}

}  // namespace

// x: projection rows holding q at off_q, k at off_k, v at off_v and the step size at off_b.
// one_token: every sequence of the batch brings exactly one row (rows == B).
US_API int us_channel_delta_prep(const void* x, long long ldx, int off_q, int off_k, int off_v,
                                 int off_b, const float* cq, const float* ck, const float* cv,
                                 const float* low, long long ldlow, const float* A_log,
                                 const float* dt_bias, void* conv, float* q, float* k, float* v,
                                 float* g, float* beta, const int* cu, const int* slots,
                                 const int* pos, int B, int rows, int H, int Hk, int D, int V, int K,
                                 int bf16, int one_token, void* stream_) {
  US_REQUIRE(low);
  ChannelPrep a{x, ldx, off_q, off_k, off_v, off_b, cq, ck, cv, low, ldlow, 0, A_log, dt_bias, conv,
                q, k, v, g, beta, cu, slots, pos, B, rows, H, Hk, D, V, K, bf16, one_token};
  return prep_impl(a, (cudaStream_t)stream_);
}

// The same for a decay per head: its argument stands at column off_a + h of the projection rows,
// dt_bias is [H] and g [rows, H].
US_API int us_head_delta_prep(const void* x, long long ldx, int off_q, int off_k, int off_v, int off_b,
                              int off_a, const float* cq, const float* ck, const float* cv,
                              const float* A_log, const float* dt_bias, void* conv, float* q, float* k,
                              float* v, float* g, float* beta, const int* cu, const int* slots,
                              const int* pos, int B, int rows, int H, int Hk, int D, int V, int K,
                              int bf16, int one_token, void* stream_) {
  ChannelPrep a{x, ldx, off_q, off_k, off_v, off_b, cq, ck, cv, nullptr, 0, off_a, A_log, dt_bias, conv,
                q, k, v, g, beta, cu, slots, pos, B, rows, H, Hk, D, V, K, bf16, one_token};
  return prep_impl(a, (cudaStream_t)stream_);
}

// out: six [rows, H, D] arrays one behind another: decay, unit key, removal, key, read-out, value.
US_API int us_general_delta_prep(const void* x, long long ldx, int off_r, int off_k, int off_v,
                                 int off_a, const float* low, long long ldlow, const float* w0,
                                 const float* a_bias, float* out, int rows, int H, int D, float rate,
                                 int bf16, void* stream_) {
  US_REQUIRE(x && low && w0 && a_bias && out && rows >= 1 && H >= 1);
  if (D < 1 || D > kMaxDim) return US_ERR_UNSUPPORTED;
  const long long warps = (long long)rows * H, n = warps * D;
  GeneralPrep a{x, ldx, off_r, off_k, off_v, off_a, low, ldlow, w0, a_bias, out, out + n, out + 2 * n,
                out + 3 * n, out + 4 * n, out + 5 * n, rows, H, D, bf16, rate};
  US_CUDA_CHECK(us::launch_pdl(general_prep_kernel, dim3((unsigned)((warps + 7) / 8)), dim3(256), 0,
                               (cudaStream_t)stream_, a));
  return US_OK;
}

// general = 0: the channel rule (g, beta); 1: the general rule (g, n, p).  q and k heads serve
// H / Hk value heads each; all vectors dense FP32.
US_API int us_vector_delta_rule(int general, const float* q, const float* k, const float* v,
                                const float* g, const float* n, const float* p, const float* beta,
                                float* state, float* out, const int* cu, const int* slots,
                                const int* pos, int B, int H, int Hk, int D, int V, void* stream_) {
  US_REQUIRE(q && k && v && g && state && out && cu && slots && pos && B >= 1 && B <= 65535);
  US_REQUIRE(general ? (n && p) : (beta != nullptr));
  US_REQUIRE(H >= 1 && Hk >= 1 && H % Hk == 0 && H <= 65535 && D >= 1 && V >= 1);
  US_REQUIRE((D & 3) || (V & 3) || (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)g | (uintptr_t)n |
               (uintptr_t)p | (uintptr_t)state) % 16) == 0);
  RuleArgs a{q, k, v, g, n, p, beta, state, out, cu, slots, pos, H, Hk, D, V};
  cudaStream_t stream = (cudaStream_t)stream_;
#define US_VD(DP) \
  if (D <= DP) return general ? launch_rule<DP, true>(a, B, stream) : launch_rule<DP, false>(a, B, stream);
  US_VD(32) US_VD(64) US_VD(128) US_VD(256)
#undef US_VD
  return US_ERR_UNSUPPORTED;
}

US_API int us_head_norm_gate(const float* o, const float* w, int w_head_stride, const void* gate,
                             long long ldg, void* y, long long ldy, int rows, int H, int V,
                             float eps, int bf16, int gate_bf16, int silu, void* stream_) {
  US_REQUIRE(o && w && gate && y && rows >= 1 && H >= 1 && V >= 1 && ldy >= (long long)H * V);
  const long long warps = (long long)rows * H;
  US_CUDA_CHECK(us::launch_pdl(head_norm_gate_kernel, dim3((unsigned)((warps + 7) / 8)), dim3(256),
                               0, (cudaStream_t)stream_, o, w, w_head_stride, gate, ldg, y, ldy, rows,
                               H, V, eps, bf16, gate_bf16, silu));
  return US_OK;
}

// One token of every sequence: projection rows x (q, k, v, step size at their columns), decay rows
// low and gate rows in, y [B, H * V] (input of the output projection) out; ring and state advance.
// US_ERR_UNSUPPORTED: the caller takes the separate kernels.
US_API int us_channel_delta_step(const void* x, long long ldx, int off_q, int off_k, int off_v,
                                 int off_b, const float* cq, const float* ck, const float* cv,
                                 const float* low, long long ldlow, const float* A_log,
                                 const float* dt_bias, void* conv, float* state, const float* nw,
                                 int nw_head_stride, const void* gate, long long ldg, void* y,
                                 long long ldy, const int* slots, const int* pos, int B, int H, int Hk,
                                 int D, int V, int K, float eps, int bf16, int gate_bf16,
                                 void* stream_) {
  US_REQUIRE(cq && ck && cv && A_log && Hk >= 1 && H % Hk == 0 && K >= 1 && (K == 1 || conv));
  if (K > kMaxTaps) return US_ERR_UNSUPPORTED;
  StepArgs a{x, ldx, off_q, off_k, off_v, off_b, cq, ck, cv, low, ldlow, 0, A_log, dt_bias, nullptr, conv,
             state, nw, nw_head_stride, gate, ldg, y, ldy, slots, pos, H, Hk, D, V, K, bf16, gate_bf16,
             0, eps, 0.f};
  return step_impl<kChannel>(a, B, (cudaStream_t)stream_);
}

// silu: the gate's activation (0: sigmoid).
US_API int us_head_delta_step(const void* x, long long ldx, int off_q, int off_k, int off_v, int off_b,
                              int off_a, const float* cq, const float* ck, const float* cv,
                              const float* A_log, const float* dt_bias, void* conv, float* state,
                              const float* nw, int nw_head_stride, const void* gate, long long ldg,
                              void* y, long long ldy, const int* slots, const int* pos, int B, int H,
                              int Hk, int D, int V, int K, float eps, int bf16, int gate_bf16, int silu,
                              void* stream_) {
  US_REQUIRE(cq && ck && cv && A_log && Hk >= 1 && H % Hk == 0 && K >= 1 && (K == 1 || conv));
  if (K > kMaxTaps) return US_ERR_UNSUPPORTED;
  StepArgs a{x, ldx, off_q, off_k, off_v, off_b, cq, ck, cv, nullptr, 0, off_a, A_log, dt_bias, nullptr, conv,
             state, nw, nw_head_stride, gate, ldg, y, ldy, slots, pos, H, Hk, D, V, K, bf16, gate_bf16,
             silu, eps, 0.f};
  return step_impl<kHead>(a, B, (cudaStream_t)stream_);
}

US_API int us_general_delta_step(const void* x, long long ldx, int off_r, int off_k, int off_v,
                                 int off_a, const float* low, long long ldlow, const float* w0,
                                 const float* a_bias, float* state, const float* nw,
                                 int nw_head_stride, const void* gate, long long ldg, void* y,
                                 long long ldy, const int* slots, const int* pos, int B, int H, int D,
                                 float rate, float eps, int bf16, int gate_bf16, void* stream_) {
  US_REQUIRE(a_bias);
  StepArgs a{x, ldx, off_r, off_k, off_v, off_a, nullptr, nullptr, nullptr, low, ldlow, 0, nullptr, w0,
             a_bias, nullptr, state, nw, nw_head_stride, gate, ldg, y, ldy, slots, pos, H, H, D, D, 1,
             bf16, gate_bf16, 0, eps, rate};
  return step_impl<kGeneral>(a, B, (cudaStream_t)stream_);
}
