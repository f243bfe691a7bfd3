// Delta rule with one decay per head (see vector_delta.cu) over packed batches, four tokens at a time:
//
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//
// With S0 the state before a block of four tokens, p_t = g_1 .. g_t and r_it = g_(i+1) .. g_t,
//
//   u_t = beta_t (v_t - p_t S0^T k_t - sum_{i < t} r_it (k_i . k_t) u_i)
//   o_t = p_t S0^T q_t + sum_{i <= t} r_it (k_i . q_t) u_i
//   S'  = p_4 S0 + sum_i r_i4 k_i u_i^T
//
// so the eight D-long reductions of a block read the same S0: they run side by side, and the chain from
// one block to the next is one reduction, four short steps and one update instead of four of each.  The
// arithmetic is FP32 throughout, and no more of it than token by token.
//
//   head_gram_kernel    the coefficients of every block and head (dots between its vectors, decays)
//   head_delta_kernel   the recurrence
//
// A CTA owns 32 value columns of one head of one sequence; a lane holds D/16 rows x 4 columns of S in
// registers as row pairs (packed FP32 instructions).  One of its columns a lane calls its own: it solves
// that one's u and hands it to the lanes that hold other rows of it.  Four warps multiply, one fetches the
// vectors of the next blocks into a ring in shared memory.  A sequence whose first packed row stands at
// position 0 starts from a zero state whatever its slot holds; a negative slot marks padding.
#include "include/us_common.cuh"
#include "include/us_f32x2.cuh"

namespace {

using namespace us::f32x2;

constexpr int kBlock = 4;         // tokens whose products share a state
constexpr int kCols = 32;         // value columns per CTA
constexpr int kCompute = 128, kCopy = 32, kThreads = kCompute + kCopy;
constexpr int kBufs = 4;          // chunks in shared memory
constexpr int kChunkBlocks = 2;   // blocks per chunk
constexpr int kMaxDim = 256;

// Coefficients of a block: beta_t | p_t | r_it k_i.k_t as 01 02 12 03 13 23 and two gaps | r_it k_i.q_t
// as [t][i] | r_i4 for i = 1 .. 3, p_4.
constexpr int kCoef = 36, kSeen = 8, kRead = 16, kCarry = 32;

struct HeadRule {
  const float *q, *k, *v;         // [rows, Hk, D] x 2, [rows, H, V]
  const float *g, *beta;          // [rows, H]
  float* coef;                    // [rows / 4 + B + 1, H, kCoef]
  float* state;                   // [slots, H, D, V]
  float* out;                     // [rows, H, V]
  const int *cu, *slots, *pos;
  int B, H, Hk, D, V;
};

// first block of sequence s among all of a batch's (one of at least a quarter of its rows each)
__device__ __forceinline__ long long first_block(int start, int s) { return (start >> 2) + s; }

// A CTA per block, a warp per key head at a time.
__global__ void __launch_bounds__(256) head_gram_kernel(const HeadRule a) {
  US_PDL_PROLOGUE();
  __shared__ float dots[8][16];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int s = 0, start = 0, n = 0, block = blockIdx.x;
  for (; s < a.B; ++s) {
    start = a.cu[s];
    n = a.cu[s + 1] - start;
    const int blocks = (n + kBlock - 1) / kBlock;
    if (block < blocks) break;
    block -= blocks;
  }
  if (s == a.B || a.slots[s] < 0) return;
  const long long row = start + block * kBlock;
  const int rows = min(kBlock, n - block * kBlock), rep = a.H / a.Hk;
  for (int hk = warp; hk < a.Hk; hk += blockDim.x >> 5) {
    float d[16];                                     // k_i . k_t for i < t (6), then k_i . q_t for i <= t
#pragma unroll
    for (int e = 0; e < 16; ++e) d[e] = 0.f;
    for (int c = lane; c < a.D; c += 32) {
      float k[kBlock], q[kBlock];
#pragma unroll
      for (int t = 0; t < kBlock; ++t) {
        const long long at = ((row + t) * a.Hk + hk) * a.D + c;
        k[t] = t < rows ? a.k[at] : 0.f;
        q[t] = t < rows ? a.q[at] : 0.f;
      }
      int e = 0;
#pragma unroll
      for (int t = 1; t < kBlock; ++t)
#pragma unroll
        for (int i = 0; i < t; ++i, ++e) d[e] = fmaf(k[i], k[t], d[e]);
#pragma unroll
      for (int t = 0; t < kBlock; ++t)
#pragma unroll
        for (int i = 0; i <= t; ++i, ++e) d[e] = fmaf(k[i], q[t], d[e]);
    }
    // sixteen sums over 32 lanes: lanes 2 e and 2 e + 1 end up with the e-th
#pragma unroll
    for (int w = 8; w >= 1; w >>= 1) {
      const bool up = lane & (2 * w);
#pragma unroll
      for (int e = 0; e < w; ++e) {
        const float keep = up ? d[e + w] : d[e], give = up ? d[e] : d[e + w];
        d[e] = keep + __shfl_xor_sync(0xffffffffu, give, 2 * w);
      }
    }
    d[0] += __shfl_xor_sync(0xffffffffu, d[0], 1);
    __syncwarp();
    if ((lane & 1) == 0) dots[warp][lane >> 1] = d[0];
    __syncwarp();
    for (int h = hk * rep; h < (hk + 1) * rep; ++h) {
      float g[kBlock], beta[kBlock];
#pragma unroll
      for (int t = 0; t < kBlock; ++t) {
        g[t] = t < rows ? a.g[(row + t) * a.H + h] : 1.f;
        beta[t] = t < rows ? a.beta[(row + t) * a.H + h] : 0.f;
      }
      auto run = [&](int i, int t) {                 // g_(i+1) .. g_t (1-based), i < t
        float r = 1.f;
#pragma unroll
        for (int x = 0; x < kBlock; ++x)
          if (x >= i && x < t) r *= g[x];
        return r;
      };
      float* out = a.coef + ((first_block(start, s) + block) * a.H + h) * kCoef;
      float v = 0.f;
      if (lane < 4) {
#pragma unroll
        for (int t = 0; t < kBlock; ++t)
          if (lane == t) v = beta[t];
      } else if (lane < kSeen) {
        v = run(0, lane - 3);
      } else if (lane < kSeen + 6) {
        const int e = lane - kSeen, t = e < 1 ? 1 : e < 3 ? 2 : 3, i = e - (t == 1 ? 0 : t == 2 ? 1 : 3);
        v = run(i + 1, t + 1) * dots[warp][e];
      } else if (lane >= kRead) {
        const int t = (lane - kRead) >> 2, i = (lane - kRead) & 3;
        if (i <= t) v = run(i + 1, t + 1) * dots[warp][6 + t * (t + 1) / 2 + i];
      }
      out[lane] = v;
      if (lane < 4) out[kCarry + lane] = lane < 3 ? run(lane + 1, kBlock) : run(0, kBlock);
    }
  }
}

template <int BYTES>
__device__ __forceinline__ void cp_async(float* dst, const float* src) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  if (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

// A block in shared memory: k of its tokens, q, 32 columns of v, the coefficients.
template <int DP>
struct Stage {
  static constexpr int kQ = kBlock * DP, kV = 2 * kBlock * DP, kC = kV + kBlock * kCols;
  static constexpr int kFloats = kC + kCoef;          // of a block
  static constexpr int kChunk = kChunkBlocks * kFloats;
};

template <int DP>
__global__ void __launch_bounds__(kThreads, DP > 128 ? 1 : 2) head_delta_kernel(const HeadRule a) {
  US_PDL_PROLOGUE();
  using St = Stage<DP>;
  constexpr int NG = DP / 64;                         // groups of four rows per lane
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, s = blockIdx.z, hk = h / (a.H / a.Hk), col0 = blockIdx.x * kCols;
  const int start = a.cu[s], T = a.cu[s + 1] - start, slot = a.slots[s];
  if (T <= 0) return;
  if (slot < 0) {                                     // padding: defined rows, no state
    for (int e = tid; e < T * kCols; e += kThreads) {
      const int t = e / kCols, c = col0 + e - t * kCols;
      if (c < a.V) a.out[((long long)(start + t) * a.H + h) * a.V + c] = 0.f;
    }
    return;
  }
  const int blocks = (T + kBlock - 1) / kBlock, chunks = (blocks + kChunkBlocks - 1) / kChunkBlocks;
  if (a.D < DP || col0 + kCols > a.V || (T % kBlock) != 0) {      // places that no copy fills: zero
    for (int e = tid; e < kBufs * St::kChunk; e += kThreads) sm[e] = 0.f;
    __syncthreads();
  }
  if (tid >= kCompute) {                              // the copying warp
    const bool quad = (a.V & 3) == 0 && (a.D & 3) == 0;
    const long long kstep = (long long)a.Hk * a.D, vstep = (long long)a.H * a.V;
    const float* kg = a.k + ((long long)start * a.Hk + hk) * a.D;
    const float* qg = a.q + ((long long)start * a.Hk + hk) * a.D;
    const float* vg = a.v + ((long long)start * a.H + h) * a.V + col0;
    const float* cg = a.coef + (first_block(start, s) * a.H + h) * kCoef;
    auto fetch = [&](int chunk) {                     // (an empty group past the end)
      for (int b = chunk * kChunkBlocks; b < min(blocks, (chunk + 1) * kChunkBlocks); ++b) {
        float* dst = sm + (chunk % kBufs) * St::kChunk + (b - chunk * kChunkBlocks) * St::kFloats;
        const int t0 = b * kBlock, n = min(kBlock, T - t0);
        if (quad) {
          for (int t = 0; t < n; ++t)
#pragma unroll
            for (int d = lane * 4; d < DP; d += 128)
              if (d < a.D) {
                cp_async<16>(dst + t * DP + d, kg + (t0 + t) * kstep + d);
                cp_async<16>(dst + St::kQ + t * DP + d, qg + (t0 + t) * kstep + d);
              }
          const int t = lane >> 3, c = (lane & 7) * 4;
          if (t < n && col0 + c < a.V) cp_async<16>(dst + St::kV + t * kCols + c, vg + (t0 + t) * vstep + c);
        } else {
          for (int t = 0; t < n; ++t) {
            for (int d = lane; d < a.D; d += 32) {
              cp_async<4>(dst + t * DP + d, kg + (t0 + t) * kstep + d);
              cp_async<4>(dst + St::kQ + t * DP + d, qg + (t0 + t) * kstep + d);
            }
            if (col0 + lane < a.V) cp_async<4>(dst + St::kV + t * kCols + lane, vg + (t0 + t) * vstep + lane);
          }
        }
        if (lane < kCoef / 4)
          cp_async<16>(dst + St::kC + lane * 4, cg + (long long)b * a.H * kCoef + lane * 4);
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll 1
    for (int r = 0; r < kBufs - 1; ++r) fetch(r);
#pragma unroll 1
    for (int r = 0; r < chunks; ++r) {
      asm volatile("cp.async.wait_group %0;" ::"n"(kBufs - 2) : "memory");
      __syncthreads();                                // chunk r is there, chunk r - 1 consumed
      fetch(r + kBufs - 1);
    }
    return;
  }
  const int kq = lane & 15;                           // lane's share of the rows
  const int own = kq >> 2, mine_t = kq & 3;           // its own column; the token whose read-out it finishes
  const int cb = warp * 8 + (lane >> 4) * 4;
  float* Sg = a.state + ((long long)slot * a.H + h) * a.D * a.V;
  const bool fresh = a.pos[start] == 0;
  // the c-th column of a lane is cb + (own ^ c): what it holds for others, they hold for it at the same c
  f2 S[NG * 2][4];                                    // row pairs x columns
#pragma unroll
  for (int j = 0; j < NG; ++j)
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int row = (j * 16 + kq) * 4 + e * 2, col = col0 + cb + (own ^ c);
        const bool in = !fresh && col < a.V;
        S[j * 2 + e][c] = pack2(in && row < a.D ? Sg[(long long)row * a.V + col] : 0.f,
                                in && row + 1 < a.D ? Sg[(long long)(row + 1) * a.V + col] : 0.f);
      }
  // sums of every column over the lanes that hold it, as far as the own column's: 4 lanes are left
  auto gather_own = [&](const f2 (&x)[kBlock][4], float (&r)[kBlock]) {
    float two[kBlock][2];
#pragma unroll
    for (int t = 0; t < kBlock; ++t)
#pragma unroll
      for (int c = 0; c < 2; ++c)
        two[t][c] = (lo2(x[t][c]) + hi2(x[t][c])) + __shfl_xor_sync(0xffffffffu, lo2(x[t][c + 2]) + hi2(x[t][c + 2]), 8);
#pragma unroll
    for (int t = 0; t < kBlock; ++t) r[t] = two[t][0] + __shfl_xor_sync(0xffffffffu, two[t][1], 4);
  };
  const bool writes = col0 + cb + own < a.V;
  float* op = a.out + ((long long)(start + mine_t) * a.H + h) * a.V + col0 + cb + own;
  const long long ostep = (long long)kBlock * a.H * a.V;
  for (int b = 0; b < blocks; ++b) {
    if (b % kChunkBlocks == 0) __syncthreads();       // this chunk's vectors are there
    const float* base = sm + (b / kChunkBlocks % kBufs) * St::kChunk + (b % kChunkBlocks) * St::kFloats;
    const float* co = base + St::kC;
    // what keys and queries see of S0
    f2 k[NG][kBlock][2], x[kBlock][4];
#pragma unroll
    for (int j = 0; j < NG; ++j) {
#pragma unroll
      for (int t = 0; t < kBlock; ++t) lds_vec(k[j][t], base + t * DP + (j * 16 + kq) * 4);
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int t = 0; t < kBlock; ++t)
#pragma unroll
          for (int c = 0; c < 4; ++c)
            x[t][c] = j + e ? fma2(S[j * 2 + e][c], k[j][t][e], x[t][c]) : mul2(S[0][c], k[0][t][0]);
    }
    float seen[kBlock];
    gather_own(x, seen);
#pragma unroll
    for (int w = 1; w < 4; w <<= 1)
#pragma unroll
      for (int t = 0; t < kBlock; ++t) seen[t] += __shfl_xor_sync(0xffffffffu, seen[t], w);
#pragma unroll
    for (int j = 0; j < NG; ++j) {
      f2 m[kBlock][2];
#pragma unroll
      for (int t = 0; t < kBlock; ++t) lds_vec(m[t], base + St::kQ + t * DP + (j * 16 + kq) * 4);
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int t = 0; t < kBlock; ++t)
#pragma unroll
          for (int c = 0; c < 4; ++c)
            x[t][c] = j + e ? fma2(S[j * 2 + e][c], m[t][e], x[t][c]) : mul2(S[0][c], m[t][0]);
    }
    // the block's writes to the own column
    const float4 be = *reinterpret_cast<const float4*>(co), p = *reinterpret_cast<const float4*>(co + 4);
    const float4 s0 = *reinterpret_cast<const float4*>(co + kSeen);
    const float2 s1 = *reinterpret_cast<const float2*>(co + kSeen + 4);
    const float4 carry = *reinterpret_cast<const float4*>(co + kCarry);
    const float* vs = base + St::kV + cb + own;
    const float u0 = be.x * fmaf(-p.x, seen[0], vs[0]);
    const float u1 = be.y * fmaf(-s0.x, u0, fmaf(-p.y, seen[1], vs[kCols]));
    const float u2 = be.z * fmaf(-s0.z, u1, fmaf(-s0.y, u0, fmaf(-p.z, seen[2], vs[2 * kCols])));
    const float u3 = be.w * fmaf(-s1.y, u2, fmaf(-s1.x, u1, fmaf(-s0.w, u0, fmaf(-p.w, seen[3], vs[3 * kCols]))));
    // S' = p_4 S0 + sum of r_i4 k_i u_i^T
    const float mine[kBlock] = {carry.x * u0, carry.y * u1, carry.z * u2, u3};
    f2 w[kBlock][4];
#pragma unroll
    for (int t = 0; t < kBlock; ++t) {
      const float w1 = __shfl_xor_sync(0xffffffffu, mine[t], 4), w2 = __shfl_xor_sync(0xffffffffu, mine[t], 8);
      const float w3 = __shfl_xor_sync(0xffffffffu, mine[t], 12);
      w[t][0] = pack2(mine[t], mine[t]);
      w[t][1] = pack2(w1, w1);
      w[t][2] = pack2(w2, w2);
      w[t][3] = pack2(w3, w3);
    }
    const f2 all = pack2(carry.w, carry.w);
#pragma unroll
    for (int j = 0; j < NG; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
#pragma unroll
        for (int c = 0; c < 4; ++c) S[j * 2 + e][c] = mul2(S[j * 2 + e][c], all);
#pragma unroll
        for (int t = 0; t < kBlock; ++t)
#pragma unroll
          for (int c = 0; c < 4; ++c) S[j * 2 + e][c] = fma2(k[j][t][e], w[t][c], S[j * 2 + e][c]);
      }
    // read-outs of the own column: four sums over the four lanes left, one each
    float q[kBlock], q2[2];
    gather_own(x, q);
    const bool hi = kq & 2, odd = kq & 1;
#pragma unroll
    for (int t = 0; t < 2; ++t)
      q2[t] = (hi ? q[t + 2] : q[t]) + __shfl_xor_sync(0xffffffffu, hi ? q[t] : q[t + 2], 2);
    float o = (odd ? q2[1] : q2[0]) + __shfl_xor_sync(0xffffffffu, odd ? q2[0] : q2[1], 1);
    const float4 rd = *reinterpret_cast<const float4*>(co + kRead + 4 * mine_t);
    o *= hi ? (odd ? p.w : p.z) : (odd ? p.y : p.x);
    o = fmaf(rd.w, u3, fmaf(rd.z, u2, fmaf(rd.y, u1, fmaf(rd.x, u0, o))));
    if (writes && b * kBlock + mine_t < T) *op = o;
    op += ostep;
  }
#pragma unroll
  for (int j = 0; j < NG; ++j)
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int row = (j * 16 + kq) * 4 + e * 2, col = col0 + cb + (own ^ c);
        if (col >= a.V) continue;
        if (row < a.D) Sg[(long long)row * a.V + col] = lo2(S[j * 2 + e][c]);
        if (row + 1 < a.D) Sg[(long long)(row + 1) * a.V + col] = hi2(S[j * 2 + e][c]);
      }
}

template <int DP>
int launch(const HeadRule& a, cudaStream_t stream) {
  constexpr int need = kBufs * Stage<DP>::kChunk * sizeof(float);
  constexpr int alone = need > 120 * 1024 ? need : 120 * 1024;      // shared memory that one CTA per SM has
  static bool configured = false;
  static int sms = 0;
  if (!configured) {
    int dev = 0;
    US_CUDA_CHECK(cudaGetDevice(&dev));
    US_CUDA_CHECK(cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev));
    US_CUDA_CHECK(cudaFuncSetAttribute(head_delta_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, alone));
    configured = true;
  }
  // CTAs that are launched while the kernel before still runs would be packed two to an SM where it
  // leaves room: with fewer CTAs than SMs each asks for more shared memory than half an SM has
  const dim3 grid(us::ceil_div(a.V, kCols), a.H, a.B);
  const size_t smem = (long long)grid.x * grid.y * grid.z <= sms ? alone : need;
  US_CUDA_CHECK(us::launch_pdl(head_delta_kernel<DP>, grid, dim3(kThreads), smem, stream, a));
  return US_OK;
}

}  // namespace

US_API long long us_head_delta_coef_floats(int rows, int B, int H) {
  return ((long long)rows / kBlock + B + 1) * H * kCoef;
}

// q and k heads serve H / Hk value heads each; all vectors dense FP32; coef: scratch of
// us_head_delta_coef_floats floats.
US_API int us_head_delta_rule(const float* q, const float* k, const float* v, const float* g,
                              const float* beta, float* coef, float* state, float* out, const int* cu,
                              const int* slots, const int* pos, int B, int rows, int H, int Hk, int D, int V,
                              void* stream_) {
  US_REQUIRE(q && k && v && g && beta && coef && state && out && cu && slots && pos && B >= 1 && B <= 65535);
  US_REQUIRE(rows >= 0 && H >= 1 && Hk >= 1 && H % Hk == 0 && H <= 65535 && D >= 1 && V >= 1);
  US_REQUIRE(((uintptr_t)coef % 16) == 0);
  US_REQUIRE((D & 3) || (V & 3) || (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) % 16) == 0);
  if (D > kMaxDim) return US_ERR_UNSUPPORTED;
  if (rows == 0) return US_OK;
  HeadRule a{q, k, v, g, beta, coef, state, out, cu, slots, pos, B, H, Hk, D, V};
  cudaStream_t stream = (cudaStream_t)stream_;
  US_CUDA_CHECK(us::launch_pdl(head_gram_kernel, dim3(rows / kBlock + B), dim3(32 * (Hk < 8 ? Hk : 8)), 0, stream, a));
  if (D <= 64) return launch<64>(a, stream);
  if (D <= 128) return launch<128>(a, stream);
  return launch<256>(a, stream);
}
