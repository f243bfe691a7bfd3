// State-space mixer with a scalar decay per head, for packed batches of sequences whose state
// lives in slots of a pool:
//
//   S <- exp(-exp(A_log) dt) S + dt B x^T,   y = S^T C + D x        S [N, V] FP32 per head
//
// or, with a fixed decay per head (linear attention: x, B, C are its values, keys and queries),
//
//   S <- decay S + B x^T,   y = S^T C
//
//   us_short_conv          causal convolution + bias + silu of x | B | C, inputs kept in a ring
//                          (without taps: silu alone)
//   us_state_space_scan    dt = softplus(raw + bias), the recurrence and its read-out
//   us_group_norm_gate     y * silu(z), RMS norm over equal parts of the row, weight; or norm and weight
//                          first, then sigmoid(z)
//   us_state_space_step    all of these for one token of every sequence in one launch
//
// A sequence whose first packed row stands at position 0 starts from a zero state whatever its
// slot holds; a negative slot marks padding.
#include "include/us_common.cuh"
#include "include/us_tc05.cuh"

namespace {

__device__ __forceinline__ float ld_any(const void* base, long long idx, int bf16) {
  return bf16 ? us::bf2f(reinterpret_cast<const __nv_bfloat16*>(base)[idx])
              : reinterpret_cast<const float*>(base)[idx];
}
__device__ __forceinline__ void st_any(void* base, long long idx, int bf16, float v) {
  if (bf16) reinterpret_cast<__nv_bfloat16*>(base)[idx] = us::f2bf(v);
  else reinterpret_cast<float*>(base)[idx] = v;
}
__device__ __forceinline__ float softplus_f(float x) {
  return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
}
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
// e^x of a decay: hundreds of factors just below one multiply along a sequence, and a biased last
// bit would add up; near zero the rounding of 1 + (e^x - 1) is the nearest one.
__device__ __forceinline__ float decay_exp(float x) { return x > -0.5f ? 1.f + expm1f(x) : expf(x); }

template <int VEC>
__device__ __forceinline__ void ld_vec(float (&o)[VEC], const void* base, long long i, int bf16) {
  if (VEC == 4 && bf16) {
    us::Pack8 p;
    p.u = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(base) + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = us::bf2f(p.b[e & 3]);
  } else if (VEC == 4) {
    const float4 v = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(base) + i);
    o[0] = v.x; o[1 % VEC] = v.y; o[2 % VEC] = v.z; o[3 % VEC] = v.w;
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = ld_any(base, i + e, bf16);
  }
}
template <int VEC>
__device__ __forceinline__ void st_vec(void* base, long long i, int bf16, const float (&v)[VEC]) {
  if (VEC == 4 && bf16) {
    us::Pack8 p;
#pragma unroll
    for (int e = 0; e < 4; ++e) p.b[e] = us::f2bf(v[e % VEC]);
    *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(base) + i) = p.u;
  } else if (VEC == 4) {
    *reinterpret_cast<float4*>(reinterpret_cast<float*>(base) + i) =
        make_float4(v[0], v[1 % VEC], v[2 % VEC], v[3 % VEC]);
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) st_any(base, i + e, bf16, v[e]);
  }
}

// ------------------------------------------------------------- convolution --
constexpr int kConvRows = 16;     // rows of one sequence per CTA
constexpr int kMaxTaps = 16;      // <= kConvRows: only a sequence's first CTA reads its ring

struct ShortConv {
  const void* x;                // projection rows
  long long ldx;
  int off;
  const float *taps, *bias;     // [C, K], [C]; null: the input itself, no bias
  void* ring;                   // [slots, K, C]: input of position p in entry p % K
  void* y;                      // [T, ldy]
  long long ldy;
  const int *cu, *slots, *pos;
  int B, T, C, K, bf16, one_token;
};

// A thread owns VEC channels over its CTA's rows, with their window in registers (KT >= K taps,
// the leading ones zero).  The CTA of a sequence's first rows reads the ring and then leaves the
// sequence's last K inputs there, so no other CTA meets it.
template <int KT, int VEC>
__global__ void __launch_bounds__(128) short_conv_kernel(const ShortConv a) {
  US_PDL_PROLOGUE();
  const int c = (blockIdx.y * 128 + threadIdx.x) * VEC;
  int tile = blockIdx.x, s, start = 0, end = 0, t0 = 0, t1 = 0;
  if (a.one_token) {
    s = start = t0 = tile;
    end = t1 = t0 + 1;
  } else {
    for (s = 0; s < a.B; ++s) {
      start = a.cu[s];
      end = a.cu[s + 1];
      const int n = (end - start + kConvRows - 1) / kConvRows;
      if (tile < n) {
        t0 = start + tile * kConvRows;
        t1 = min(end, t0 + kConvRows);
        break;
      }
      tile -= n;
    }
  }
  if (t0 == t1 || c >= a.C) return;
  const int slot = a.slots[s], p0 = a.pos[start];
  const long long ring = (long long)max(slot, 0) * a.K * a.C + c;
  float w[KT][VEC], win[KT][VEC], b[VEC];
#pragma unroll
  for (int j = 0; j < KT; ++j) {
    const int k = j - (KT - a.K);
#pragma unroll
    for (int e = 0; e < VEC; ++e) w[j][e] = k < 0 ? 0.f : a.taps ? a.taps[(long long)(c + e) * a.K + k] : 1.f;
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) b[e] = a.bias ? a.bias[c + e] : 0.f;
#pragma unroll
  for (int j = 1; j < KT; ++j) {                    // inputs of the rows before t0
    const int back = KT - j, src = t0 - back, p = p0 + src - start;
#pragma unroll
    for (int e = 0; e < VEC; ++e) win[j][e] = 0.f;
    if (back < a.K) {
      if (src >= start) ld_vec<VEC>(win[j], a.x, (long long)src * a.ldx + a.off + c, a.bf16);
      else if (p >= 0 && slot >= 0) ld_vec<VEC>(win[j], a.ring, ring + (long long)(p % a.K) * a.C, a.bf16);
    }
  }
  for (int t = t0; t < t1; ++t) {
#pragma unroll
    for (int j = 0; j + 1 < KT; ++j)
#pragma unroll
      for (int e = 0; e < VEC; ++e) win[j][e] = win[j + 1][e];
    ld_vec<VEC>(win[KT - 1], a.x, (long long)t * a.ldx + a.off + c, a.bf16);
    float y[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      float acc = b[e];
#pragma unroll
      for (int j = 0; j < KT; ++j) acc = fmaf(w[j][e], win[j][e], acc);
      y[e] = silu_f(acc);
    }
    st_vec<VEC>(a.y, (long long)t * a.ldy + c, a.bf16, y);
  }
  if (t0 > start || slot < 0 || a.K == 1) return;
  for (int t = max(start, end - a.K); t < end; ++t) {
    float v[VEC];
    ld_vec<VEC>(v, a.x, (long long)t * a.ldx + a.off + c, a.bf16);
    st_vec<VEC>(a.ring, ring + (long long)((p0 + t - start) % a.K) * a.C, a.bf16, v);
  }
}

// -------------------------------------------------------------- recurrence --
struct ScanArgs {
  const void* u;                // [T, ldu]: x (H * V) | B (G * N) | C (G * N)
  long long ldu;
  const void* dt;               // raw step sizes, column h of rows at lddt
  long long lddt;
  const float *dt_bias, *A_log, *D;   // [H]
  const double* log_decay;      // [H] or null; else no step sizes and no D
  float* state;                 // [slots, H, N, V]
  void* y;                      // [T, ldy]
  long long ldy;
  const int *cu, *slots, *pos;
  int T, H, V, N, G, bf16;
};

constexpr int kCols = 32;       // state columns per CTA
constexpr int kChunk = 16;      // tokens staged per round

// Token by token, any sizes, both types: a CTA owns 32 columns of one head of one sequence, a lane
// NP / 4 rows of one column.
template <int NP>
__global__ void __launch_bounds__(128) scan_rows_kernel(const ScanArgs a) {
  US_PDL_PROLOGUE();
  constexpr int kPer = NP / 4;
  __shared__ __align__(16) float Bs[kChunk][NP], Cs[kChunk][NP];
  __shared__ float xs[kChunk][kCols], ys[kChunk][kCols], dts[kChunk], dec[kChunk];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, vl = lane >> 2, kq = lane & 3;
  const int h = blockIdx.y, s = blockIdx.z, g = h / (a.H / a.G);
  const int col = blockIdx.x * kCols + warp * 8 + vl;
  const int start = a.cu[s], T = a.cu[s + 1] - start, slot = a.slots[s];
  if (T <= 0) return;
  if (slot < 0) {
    for (int e = tid; e < T * kCols; e += 128) {
      const int c = blockIdx.x * kCols + e % kCols;
      if (c < a.V) st_any(a.y, (long long)(start + e / kCols) * a.ldy + (long long)h * a.V + c, a.bf16, 0.f);
    }
    return;
  }
  const bool fresh = a.pos[start] == 0, col_ok = col < a.V;
  float* Sg = a.state + ((long long)slot * a.H + h) * a.N * a.V;
  const bool fixed = a.log_decay != nullptr;
  const float A = fixed ? 0.f : expf(a.A_log[h]), D = fixed ? 0.f : a.D[h], bias = fixed ? 0.f : a.dt_bias[h];
  const float decay = fixed ? (float)exp(a.log_decay[h]) : 0.f;
  const long long ob = (long long)a.H * a.V + (long long)g * a.N, oc = ob + (long long)a.G * a.N;
  float S[kPer];
#pragma unroll
  for (int j = 0; j < kPer; ++j) {
    const int row = ((j >> 2) * 4 + kq) * 4 + (j & 3);
    S[j] = (!fresh && col_ok && row < a.N) ? Sg[(long long)row * a.V + col] : 0.f;
  }
  for (int c0 = 0; c0 < T; c0 += kChunk) {
    const int n = min(kChunk, T - c0);
    __syncthreads();
    for (int e = tid; e < n * NP; e += 128) {
      const int t = e / NP, i = e - t * NP;
      const long long row = (long long)(start + c0 + t) * a.ldu;
      Bs[t][i] = i < a.N ? ld_any(a.u, row + ob + i, a.bf16) : 0.f;
      Cs[t][i] = i < a.N ? ld_any(a.u, row + oc + i, a.bf16) : 0.f;
    }
    for (int e = tid; e < n * kCols; e += 128) {
      const int t = e / kCols, c = blockIdx.x * kCols + e % kCols;
      xs[t][e % kCols] = c < a.V ? ld_any(a.u, (long long)(start + c0 + t) * a.ldu + (long long)h * a.V + c, a.bf16) : 0.f;
    }
    if (fixed) {
      if (tid < n) {
        dts[tid] = 1.f;
        dec[tid] = decay;
      }
    } else if (tid < n) {
      const float dt = softplus_f(ld_any(a.dt, (long long)(start + c0 + tid) * a.lddt + h, a.bf16) + bias);
      dts[tid] = dt;
      dec[tid] = decay_exp(-A * dt);
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float e = dec[t], x = xs[t][warp * 8 + vl], dx = dts[t] * x;
      float o = 0.f;
#pragma unroll
      for (int j = 0; j < kPer / 4; ++j) {
        const float4 b4 = *reinterpret_cast<const float4*>(&Bs[t][(j * 4 + kq) * 4]);
        const float4 c4 = *reinterpret_cast<const float4*>(&Cs[t][(j * 4 + kq) * 4]);
        S[j * 4] = fmaf(S[j * 4], e, b4.x * dx);
        S[j * 4 + 1] = fmaf(S[j * 4 + 1], e, b4.y * dx);
        S[j * 4 + 2] = fmaf(S[j * 4 + 2], e, b4.z * dx);
        S[j * 4 + 3] = fmaf(S[j * 4 + 3], e, b4.w * dx);
        o += S[j * 4] * c4.x + S[j * 4 + 1] * c4.y + S[j * 4 + 2] * c4.z + S[j * 4 + 3] * c4.w;
      }
      o += __shfl_xor_sync(0xffffffffu, o, 1);
      o += __shfl_xor_sync(0xffffffffu, o, 2);
      if (kq == 0) ys[t][warp * 8 + vl] = fmaf(D, x, o);
    }
    __syncthreads();
    for (int e = tid; e < n * kCols; e += 128) {
      const int t = e / kCols, c = blockIdx.x * kCols + e % kCols;
      if (c < a.V) st_any(a.y, (long long)(start + c0 + t) * a.ldy + (long long)h * a.V + c, a.bf16, ys[t][e % kCols]);
    }
  }
  if (!col_ok) return;
#pragma unroll
  for (int j = 0; j < kPer; ++j) {
    const int row = ((j >> 2) * 4 + kq) * 4 + (j & 3);
    if (row < a.N) Sg[(long long)row * a.V + col] = S[j];
  }
}

// --------------------------------------------------------- gate, group norm --
// A CTA per (row, part).  NV > 0: the part stays in registers; 0: it is read twice.
template <int NV, int VEC>
__global__ void __launch_bounds__(256)
group_norm_gate_kernel(const void* __restrict__ y, long long ldy, const void* __restrict__ z,
                       long long ldz, int groups, const float* __restrict__ w, void* __restrict__ out,
                       long long ldo, int n, float eps, int bf16, int z_bf16,
                       int after, long long padded) {
  US_PDL_PROLOGUE();
  __shared__ float part[8];
  const int len = n / groups, g = blockIdx.y, step = blockDim.x * VEC, c0 = threadIdx.x * VEC;
  const long long yi = (long long)blockIdx.x * ldy + (long long)g * len;
  const long long zi = (long long)blockIdx.x * ldz + (long long)g * len;
  const long long oi = (long long)blockIdx.x * ldo + (long long)g * len;
  auto gated = [&](int c, float (&v)[VEC]) {
    float gz[VEC];
    ld_vec<VEC>(v, y, yi + c, bf16);
    if (after) return;
    ld_vec<VEC>(gz, z, zi + c, z_bf16);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] *= silu_f(gz[e]);
  };
  auto put = [&](int c, float (&v)[VEC], float inv) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] *= inv * w[g * len + c + e];
    if (after) {
      float gz[VEC];
      ld_vec<VEC>(gz, z, zi + c, z_bf16);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] *= sigmoid_f(gz[e]);
    }
    st_vec<VEC>(out, oi + c, bf16, v);
  };
  float held[NV > 0 ? NV : 1][VEC], ss = 0.f;
  if (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      if (c >= len) continue;
      gated(c, held[i]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += held[i][e] * held[i][e];
    }
  } else {
    for (int c = c0; c < len; c += step) {
      gated(c, held[0]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += held[0][e] * held[0][e];
    }
  }
  ss = us::warp_sum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int k = 0; k < (int)(blockDim.x >> 5); ++k) ss += part[k];
  const float inv = 1.f / sqrtf(ss / (float)len + eps);
  if (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (c0 + i * step < len) put(c0 + i * step, held[i], inv);
  } else {
    for (int c = c0; c < len; c += step) {
      gated(c, held[0]);
      put(c, held[0], inv);
    }
  }
  if (g == groups - 1)
    for (long long c = n + threadIdx.x; c < padded; c += blockDim.x)
      st_any(out, (long long)blockIdx.x * ldo + c, bf16, 0.f);
}

// ------------------------------------------------------------- decode step --
struct StepArgs {
  const void* x;                // projection rows: z | x B C | dt at the three offsets
  long long ldx;
  int oz, oc, odt;
  const float *taps, *bias;     // [C, K], [C]; null: the input itself, no bias
  void* ring;                   // [slots, K, C]
  const float *dt_bias, *A_log, *D, *w;   // [H] x 3, [H * V]
  const double* log_decay;      // [H] or null; else no step sizes and no D
  float* state;                 // [slots, H, N, V]
  void* out;                    // [B, ldo]
  long long ldo;
  const int *slots, *pos;
  int H, V, N, G, K, bf16, heads;         // heads: of a norm part (the cluster), 0: no gate and norm
  int after;                    // gate: silu before the norm (0) or sigmoid after it (1)
  float eps;
};

constexpr int kStepThreads = 256;

// One CTA per (head, sequence).  A thread keeps up to R rows of four state columns (VQ threads
// span the columns); their loads are issued first, the convolution, the step size and the decay are
// formed meanwhile.  B and C of a group are convolved by each of its heads and kept by the
// first one (the entry that a token writes is none of those it reads).  The heads of a norm part are
// one cluster that adds up their sums of squares.
template <int VQ, int R>
__global__ void __launch_bounds__(kStepThreads, R <= 8 ? 3 : 2) state_space_step_kernel(const StepArgs a) {
  US_PDL_PROLOGUE();
  constexpr int GR = kStepThreads / VQ;           // row groups
  extern __shared__ __align__(16) float sm[];
  float* u = sm;                                  // [V | N | N] convolved inputs
  float* red = u + ((a.V + 2 * a.N + 3) & ~3);    // [GR][VQ * 4]
  __shared__ float part[33], steps[2], total;
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int g = h / (a.H / a.G), inner = a.H * a.V, C = inner + 2 * a.G * a.N;
  const int slot = a.slots[b], p = a.pos[b];
  const bool live = slot >= 0;
  const int q = tid % VQ, gr = tid / VQ, v0 = q * 4;
  float* Sg = a.state + ((long long)max(slot, 0) * a.H + h) * a.N * a.V;
  float4 S[R];
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int row = gr + j * GR;
    S[j] = (live && p > 0 && row < a.N && v0 < a.V)
               ? __ldcs(reinterpret_cast<const float4*>(Sg + (long long)row * a.V + v0))
               : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const bool mine = tid < a.V;                    // thread v < V finishes column v
  const float z = live && mine && a.heads > 0
                      ? ld_any(a.x, (long long)b * a.ldx + a.oz + (long long)h * a.V + tid, a.bf16) : 0.f;
  if (live) {
    const bool keeps = h % (a.H / a.G) == 0;      // this head writes its group's B and C inputs
    for (int e = tid; e < a.V + 2 * a.N; e += kStepThreads) {
      const int c = e < a.V ? h * a.V + e
                            : inner + (e < a.V + a.N ? g * a.N + e - a.V : (a.G + g) * a.N + e - a.V - a.N);
      const float now = ld_any(a.x, (long long)b * a.ldx + a.oc + c, a.bf16);
      const float* w = a.taps + (long long)c * a.K;
      float acc = a.taps ? fmaf(w[a.K - 1], now, a.bias ? a.bias[c] : 0.f) : now;
      for (int k = 1; k < min(a.K, p + 1); ++k)
        acc = fmaf(w[a.K - 1 - k], ld_any(a.ring, ((long long)slot * a.K + (p - k) % a.K) * C + c, a.bf16), acc);
      if (a.K > 1 && (e < a.V || keeps))
        st_any(a.ring, ((long long)slot * a.K + p % a.K) * C + c, a.bf16, now);
      acc = silu_f(acc);
      u[e] = a.bf16 ? us::bf2f(us::f2bf(acc)) : acc;
    }
    if (tid == kStepThreads - 1 && a.log_decay) {
      steps[0] = 1.f;
      steps[1] = (float)exp(a.log_decay[h]);
    } else if (tid == kStepThreads - 1) {
      const float dt = softplus_f(ld_any(a.x, (long long)b * a.ldx + a.odt + h, a.bf16) + a.dt_bias[h]);
      steps[0] = dt;
      steps[1] = decay_exp(-expf(a.A_log[h]) * dt);
    }
  }
  __syncthreads();
  float y = 0.f;
  if (live) {
    const float dt = steps[0], dec = steps[1];
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (v0 < a.V) {
      const float4 x4 = make_float4(u[v0] * dt, u[v0 + 1] * dt, u[v0 + 2] * dt, u[v0 + 3] * dt);
#pragma unroll
      for (int j = 0; j < R; ++j) {
        const int row = gr + j * GR;
        if (row >= a.N) continue;
        const float B = u[a.V + row], Cn = u[a.V + a.N + row];
        S[j].x = fmaf(S[j].x, dec, B * x4.x);
        S[j].y = fmaf(S[j].y, dec, B * x4.y);
        S[j].z = fmaf(S[j].z, dec, B * x4.z);
        S[j].w = fmaf(S[j].w, dec, B * x4.w);
        __stcs(reinterpret_cast<float4*>(Sg + (long long)row * a.V + v0), S[j]);
        o.x = fmaf(S[j].x, Cn, o.x);
        o.y = fmaf(S[j].y, Cn, o.y);
        o.z = fmaf(S[j].z, Cn, o.z);
        o.w = fmaf(S[j].w, Cn, o.w);
      }
    }
    *reinterpret_cast<float4*>(red + (gr * VQ + q) * 4) = o;
  }
  __syncthreads();
  if (live && mine) {
    for (int r = 0; r < GR; ++r) y += red[r * VQ * 4 + tid];
    if (!a.log_decay) y = fmaf(a.D[h], u[tid], y);
    if (a.bf16) y = us::bf2f(us::f2bf(y));
  }
  const long long at = (long long)b * a.ldo + (long long)h * a.V + tid;
  if (a.heads == 0) {
    if (mine) st_any(a.out, at, a.bf16, y);
    return;
  }
  if (!a.after) y *= silu_f(z);
  float ss = us::block_sum(y * y, part);
  if (a.heads > 1) {
    if (tid == 0) total = ss;
    tc::cluster_sync();
    const uint32_t addr = (uint32_t)__cvta_generic_to_shared(&total);
    ss = 0.f;
    for (int r = 0; r < a.heads; ++r) ss += tc::ld_dsmem_f32(tc::map_to_cta(addr, r));
  }
  if (mine) {
    if (a.after) y *= sigmoid_f(z);
    st_any(a.out, at, a.bf16,
           live ? y * (1.f / sqrtf(ss / (float)(max(a.heads, 1) * a.V) + a.eps)) * a.w[h * a.V + tid] : 0.f);
  }
  if (a.heads > 1) tc::cluster_sync();            // nobody leaves while its sum may still be read
}

template <int VQ, int R>
int launch_step_rows(const StepArgs& a, int B, cudaStream_t stream) {
  const size_t smem = (((a.V + 2 * a.N + 3) & ~3) + kStepThreads * 4) * sizeof(float);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(a.H, B);
  cfg.blockDim = dim3(kStepThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = us::pdl_enabled() ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = a.heads;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = a.heads > 1 ? 2 : 1;
  US_CUDA_CHECK(cudaLaunchKernelEx(&cfg, state_space_step_kernel<VQ, R>, a));
  return US_OK;
}

template <int VQ>
int launch_step(const StepArgs& a, int B, cudaStream_t stream) {
  const int rows = us::ceil_div(a.N, kStepThreads / VQ);
  return rows <= 4 ? launch_step_rows<VQ, 4>(a, B, stream)
                   : rows <= 8 ? launch_step_rows<VQ, 8>(a, B, stream) : launch_step_rows<VQ, 16>(a, B, stream);
}

bool aligned(const void* p, int bytes) { return ((uintptr_t)p % bytes) == 0; }

}  // namespace

US_API int us_short_conv(const void* x, long long ldx, int off, const float* taps, const float* bias,
                         void* ring, void* y, long long ldy, const int* cu, const int* slots,
                         const int* pos, int B, int T, int C, int K, int bf16, int one_token,
                         void* stream_) {
  US_REQUIRE(x && y && cu && slots && pos && B >= 1 && T >= 0 && C >= 1 && K >= 1 && (taps || K == 1));
  US_REQUIRE((K == 1 || ring) && (!one_token || B == T));
  if (K > kMaxTaps) return US_ERR_LIMIT;
  if (T == 0) return US_OK;
  ShortConv a{x, ldx, off, taps, bias, ring, y, ldy, cu, slots, pos, B, T, C, K, bf16, one_token};
  const int bytes = bf16 ? 8 : 16;
  const bool vec = (C % 4) == 0 && (off % 4) == 0 && (ldx % 4) == 0 && (ldy % 4) == 0 &&
                   aligned(x, bytes) && aligned(y, bytes) && aligned(ring, bytes);
  const dim3 grid(one_token ? T : T / kConvRows + B, us::ceil_div(C, 128 * (vec ? 4 : 1)));
#define US_CONV(KT, VEC)                                                                           \
  US_CUDA_CHECK(us::launch_pdl(short_conv_kernel<KT, VEC>, grid, dim3(128), 0, (cudaStream_t)stream_, a))
  if (vec) {
    if (K <= 4) US_CONV(4, 4);
    else if (K <= 8) US_CONV(8, 4);
    else US_CONV(16, 4);
  } else {
    if (K <= 4) US_CONV(4, 1);
    else if (K <= 8) US_CONV(8, 1);
    else US_CONV(16, 1);
  }
#undef US_CONV
  return US_OK;
}

US_API int us_state_space_scan(const void* u, long long ldu, const void* proj, long long ldp,
                               int off_dt, const float* dt_bias, const float* A_log, const float* D,
                               const double* log_decay, float* state, void* y, long long ldy,
                               const int* cu, const int* slots, const int* pos, int B, int T, int H,
                               int V, int N, int G, int bf16, void* stream_) {
  US_REQUIRE(u && (log_decay || (proj && dt_bias && A_log && D)) && state && y && cu && slots && pos);
  US_REQUIRE(B >= 1 && T >= 0 && H >= 1 && V >= 1 && N >= 1 && G >= 1 && H % G == 0);
  if (T == 0) return US_OK;
  const void* dt = bf16 ? (const void*)((const __nv_bfloat16*)proj + off_dt)
                        : (const void*)((const float*)proj + off_dt);
  ScanArgs a{u, ldu, dt, ldp, dt_bias, A_log, D, log_decay, state, y, ldy, cu, slots, pos, T, H, V, N, G, bf16};
  const dim3 grid(us::ceil_div(V, kCols), H, B);
#define US_SCAN(NP)                                                                                \
  US_CUDA_CHECK(us::launch_pdl(scan_rows_kernel<NP>, grid, dim3(128), 0, (cudaStream_t)stream_, a))
  if (N <= 16) US_SCAN(16);
  else if (N <= 32) US_SCAN(32);
  else if (N <= 64) US_SCAN(64);
  else if (N <= 128) US_SCAN(128);
  else if (N <= 256) US_SCAN(256);
  else return US_ERR_LIMIT;
#undef US_SCAN
  return US_OK;
}

// Columns n .. padded of an output row become zero.
US_API int us_group_norm_gate(const void* y, long long ldy, const void* z, long long ldz, int groups,
                              const float* w, void* out, long long ldo, int padded, int T, int n,
                              int bf16, float eps, int z_bf16, int after, void* stream_) {
  US_REQUIRE(y && z && w && out && T >= 0 && n >= 1 && groups >= 1 && n % groups == 0 && padded >= n &&
             ldo >= padded);
  if (T == 0) return US_OK;
  const int len = n / groups, yb = bf16 ? 8 : 16, zb = z_bf16 ? 8 : 16;
  const bool vec = (len % 4) == 0 && (ldy % 4) == 0 && (ldz % 4) == 0 && (ldo % 4) == 0 &&
                   aligned(y, yb) && aligned(z, zb) && aligned(out, yb);
  const int per = vec ? 4 : 1, threads = min(256, us::ceil_div(us::ceil_div(len, per), 32) * 32);
  const int nv = us::ceil_div(len, threads * per);
  const dim3 grid(T, groups);
#define US_GN(NV, VEC)                                                                             \
  US_CUDA_CHECK(us::launch_pdl(group_norm_gate_kernel<NV, VEC>, grid, dim3(threads), 0,             \
                               (cudaStream_t)stream_, y, ldy, z, ldz, groups, w, out, ldo, n, eps,  \
                               bf16, z_bf16, after, (long long)padded))
  if (vec) {
    if (nv <= 1) US_GN(1, 4);
    else if (nv <= 2) US_GN(2, 4);
    else if (nv <= 4) US_GN(4, 4);
    else if (nv <= 8) US_GN(8, 4);
    else US_GN(0, 4);
  } else {
    if (nv <= 4) US_GN(4, 1);
    else US_GN(0, 1);
  }
#undef US_GN
  return US_OK;
}

// One token of every sequence: convolution, recurrence, read-out and, with heads >= 1 (the heads of a
// norm part, at most 8, dividing H), gate and norm.  V a multiple of 4, V <= 256, N <= 16 row groups.
US_API int us_state_space_step(const void* x, long long ldx, int oz, int oc, int odt,
                               const float* taps, const float* bias, void* ring,
                               const float* dt_bias, const float* A_log, const float* D,
                               const double* log_decay, const float* w, float* state, void* out,
                               long long ldo, const int* slots, const int* pos, int B, int H, int V,
                               int N, int G, int K, int bf16, int heads, int after, float eps,
                               void* stream_) {
  US_REQUIRE(x && (taps || K == 1) && (log_decay || (dt_bias && A_log && D)) && state && out && slots && pos);
  US_REQUIRE(B >= 0 && H >= 1 && V >= 4 && N >= 1 && G >= 1 && H % G == 0 && K >= 1 && (K == 1 || ring) &&
             (V % 4) == 0 && heads >= 0 && heads <= 8 && (heads == 0 || (H % heads == 0 && w)) && B <= 65535);
  const int vq = V <= 32 ? 8 : V <= 64 ? 16 : V <= 128 ? 32 : 64;
  if (V > 256 || us::ceil_div(N, kStepThreads / vq) > 16) return US_ERR_LIMIT;
  if (B == 0) return US_OK;
  StepArgs a{x, ldx, oz, oc, odt, taps, bias, ring, dt_bias, A_log, D, w, log_decay, state, out, ldo, slots, pos,
             H, V, N, G, K, bf16, heads, after, eps};
  cudaStream_t stream = (cudaStream_t)stream_;
  switch (vq) {
    case 8: return launch_step<8>(a, B, stream);
    case 16: return launch_step<16>(a, B, stream);
    case 32: return launch_step<32>(a, B, stream);
    default: return launch_step<64>(a, B, stream);
  }
}
