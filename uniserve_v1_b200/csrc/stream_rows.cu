// Rows of the FP32 residual stream between two sublayers, in one launch:
//
//   source   r(t) = rms(embed[id] * scale + table2[row]) * w              start of the stream
//            r(t) = residual(t) + rms(y(t)) * w                           output norm and add
//            r(t) = embed[id] * scale,  residual(t) + gain * y(t)         without w (plain form)
//            r(t) = embed[id] * scale,  residual(t) + ln(y(t)) * w + b    layer form
//   output   h(t) = rms(r(t)) * w_out                                     input norm
//            h(t) = r(t)   or   ln(r(t)) * w_out + b_out                  layer form
//            x(t) = h(t)   or   h(t) + (h(t - 1) - h(t)) * mu             token shift
//
// In the plain and the layer form y may also be a mixture of experts: sum_k weight_k * (row perm_k of the
// expert rows, or row t of `ident` for an expert without tensors, perm_k < 0) + shared(t), the last one
// times sigmoid(shared_gate(t)) in the layer form.
//
// with rms(v) = v / sqrt(mean(v^2) + eps) and ln(v) = (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps).  r goes to a second residual buffer (the one that is
// read stays as it is), because a shifted row needs its neighbour's h: a CTA takes up to kRows
// consecutive rows of one sequence and forms the row before its first one itself.  The h before a
// sequence's first row of the batch comes from the state slot; the CTA that reads it also forms
// the h of the sequence's last row and stores it there, so no other CTA meets the slot.
//
//   bigram_rows   table rows hashed from a token and the one before it (its own slot of state)
//   poly_norm     a N(z) + b N(z^2) + c N(z^3) + e,  N(v) = v / sqrt(mean(v^2) + eps) over the row
//
// Rows are padded to a multiple of 8 columns with zeros; `width` is the true column count.
// Element types: 1 = bf16, 0 = fp32.  All arithmetic is FP32.
#include "include/us_common.cuh"

namespace {

constexpr int kRows = 8;          // rows of a sequence per CTA

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
__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float4 mul4(float4 a, float4 b, float s) {
  return make_float4(a.x * s * b.x, a.y * s * b.y, a.z * s * b.z, a.w * s * b.w);
}
__device__ __forceinline__ float4 add4(float4 a, float4 b) {
  return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w);
}
__device__ __forceinline__ float4 mix4(float4 h, float4 before, float4 mu) {
  return make_float4(h.x + (before.x - h.x) * mu.x, h.y + (before.y - h.y) * mu.y,
                     h.z + (before.z - h.z) * mu.z, h.w + (before.w - h.w) * mu.w);
}

// Sum over the block; `buf` holds 2 x 32 floats used in turns, so one barrier per sum suffices.
__device__ __forceinline__ float turn_sum(float v, float* buf, int& turn) {
  v = us::warp_sum(v);
  float* b = buf + (turn ^= 32);
  if ((threadIdx.x & 31) == 0) b[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) s += b[w];
  return s;
}

struct StreamRows {
  const int *ids, *rows2;     // start of the stream: token ids, rows of the second table (or null)
  const void *table, *table2;
  float scale;
  int vocab, n2;
  const void* y;              // [T, W] sublayer output (null: start of the stream)
  const float* residual;      // [T, W]
  const float* w;             // [W], null: plain form
  float* residual_out;        // [T, W]
  const float* w_out;         // [W]
  const float* mu;            // [W] or null: no token shift
  float* state;               // [slots, W]: h of a sequence's last token
  const int *cu, *slots, *pos;
  void* x;                    // [T, W]
  int B, T, W, width, bf16, one_token;
  float eps;
  int rows;                   // rows per CTA without a shift
  unsigned int* status;
  // plain form
  float gain;
  const void* y_perm;         // expert rows, or null: y
  const int* perm;            // [T, top]
  const float* route_w;       // [T, top]
  int top;
  const void *ident, *shared; // [T, W] or null
  // layer form
  const float *b, *b_out;     // [W]
  const float* shared_gate;   // logit of row t at t * ld_gate, or null: the shared rows as they are
  long long ld_gate;
};

enum Form : int { kOutNorm = 0, kPlain = 1, kLayer = 2 };

template <int NV, int FORM, bool MIX>
__global__ void __launch_bounds__(256, NV <= 2 ? 4 : 1) stream_rows_kernel(const StreamRows a) {
  US_PDL_PROLOGUE();
  __shared__ float buf[64];
  int turn = 0;
  const int W = a.W, step = blockDim.x * 4, c0 = threadIdx.x * 4;
  const float inv_n = 1.f / (float)a.width;
  // rows of this CTA: t0 .. t1 of sequence s
  int s = -1, t0, t1, start = 0, end = 0;
  if (!a.mu) {
    t0 = blockIdx.x * a.rows;
    t1 = min(a.T, t0 + a.rows);
  } else if (a.one_token) {
    s = start = t0 = blockIdx.x;
    end = t1 = t0 + 1;
  } else {
    int tile = blockIdx.x;
    t0 = t1 = 0;
    for (s = 0; s < a.B; ++s) {
      start = a.cu[s];
      end = a.cu[s + 1];
      const int n = (end - start + kRows - 1) / kRows;
      if (tile < n) {
        t0 = start + tile * kRows;
        t1 = min(end, t0 + kRows);
        break;
      }
      tile -= n;
    }
    if (t0 == t1) return;
  }
  // a mixture's routes of a row (lane k: expert k) and the shared rows' gate, fetched a row ahead
  int next_p = -1;
  float next_w = 0.f, next_g = 1.f;
  auto routes = [&](int t) {
    const int lane = threadIdx.x & 31;
    if (t >= t1) return;
    if (lane < a.top) {
      next_p = a.perm[(long long)t * a.top + lane];
      next_w = a.route_w[(long long)t * a.top + lane];
    }
    if (FORM == kLayer && a.shared_gate) next_g = 1.f / (1.f + expf(-a.shared_gate[t * a.ld_gate]));
  };
  if constexpr (MIX) routes(t0);
  // raw operands of a row: the sublayer's output (or the embedding sum) and the residual
  auto load = [&](int t, float4 (&v)[NV], float4 (&r)[NV]) {
    const long long base = (long long)t * W;
    if constexpr (MIX) {
      const int p_row = next_p;
      const float w_row = next_w, sg = next_g;
      routes(t + 1);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * step;
        v[i] = r[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= W) continue;
        if (a.shared) v[i] = ld4(a.shared, base + c, a.bf16);
        if (FORM == kLayer) v[i] = make_float4(v[i].x * sg, v[i].y * sg, v[i].z * sg, v[i].w * sg);
        r[i] = *reinterpret_cast<const float4*>(a.residual + base + c);
      }
#pragma unroll 4
      for (int k = 0; k < a.top; ++k) {
        const int p = __shfl_sync(0xffffffffu, p_row, k);
        const float wk = __shfl_sync(0xffffffffu, w_row, k);
        if (p < 0 && !a.ident) continue;
        const void* from = p < 0 ? a.ident : a.y_perm;
        const long long row = (long long)(p < 0 ? t : p) * W;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = c0 + i * step;
          if (c >= W) continue;
          const float4 e = ld4(from, row + c, a.bf16);
          v[i] = make_float4(fmaf(wk, e.x, v[i].x), fmaf(wk, e.y, v[i].y), fmaf(wk, e.z, v[i].z),
                             fmaf(wk, e.w, v[i].w));
        }
      }
    } else if (a.y) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * step;
        v[i] = r[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= W) continue;
        v[i] = ld4(a.y, base + c, a.bf16);
        r[i] = *reinterpret_cast<const float4*>(a.residual + base + c);
      }
    } else {
      const int id = a.ids[t], r2 = a.rows2 ? a.rows2[t] : 0;
      const bool ok = id >= 0 && id < a.vocab && r2 >= 0 && (!a.rows2 || r2 < a.n2);
      if (!ok && threadIdx.x == 0) us_dev_fail(a.status, US_DEV_BOUNDS);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = c0 + i * step;
        v[i] = r[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (ok && c < W) {
          const float4 e = ld4(a.table, (long long)id * W + c, a.bf16);
          v[i] = make_float4(e.x * a.scale, e.y * a.scale, e.z * a.scale, e.w * a.scale);
          if (a.rows2) v[i] = add4(v[i], ld4(a.table2, (long long)r2 * W + c, a.bf16));
        }
      }
    }
  };
  auto layer = [&](float4 (&v)[NV], const float* w, const float* b) {
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) sum += v[i].x + v[i].y + v[i].z + v[i].w;      // columns past `width` are zero
    const float mean = turn_sum(sum, buf, turn) * inv_n;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      v[i] = make_float4(c < a.width ? v[i].x - mean : 0.f, c + 1 < a.width ? v[i].y - mean : 0.f,
                         c + 2 < a.width ? v[i].z - mean : 0.f, c + 3 < a.width ? v[i].w - mean : 0.f);
      ss += sq4(v[i]);
    }
    const float inv = 1.f / sqrtf(turn_sum(ss, buf, turn) * inv_n + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      if (c < W)
        v[i] = add4(mul4(v[i], *reinterpret_cast<const float4*>(w + c), inv), *reinterpret_cast<const float4*>(b + c));
    }
  };
  auto source = [&](float4 (&v)[NV], const float4 (&r)[NV]) {     // v becomes the row of the stream
    if (FORM == kLayer) {
      if (!a.residual) return;                   // start of the stream
      layer(v, a.w, a.b);
#pragma unroll
      for (int i = 0; i < NV; ++i) v[i] = add4(r[i], v[i]);
      return;
    }
    if (FORM == kPlain) {
#pragma unroll
      for (int i = 0; i < NV; ++i)
        v[i] = make_float4(fmaf(a.gain, v[i].x, r[i].x), fmaf(a.gain, v[i].y, r[i].y),
                           fmaf(a.gain, v[i].z, r[i].z), fmaf(a.gain, v[i].w, r[i].w));
      return;
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) ss += sq4(v[i]);
    const float inv = 1.f / sqrtf(turn_sum(ss, buf, turn) * inv_n + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      if (c < W) v[i] = add4(r[i], mul4(v[i], *reinterpret_cast<const float4*>(a.w + c), inv));
    }
  };
  auto norm = [&](float4 (&v)[NV]) {
    if (FORM == kLayer) {
      if (a.w_out) layer(v, a.w_out, a.b_out);
      return;
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) ss += sq4(v[i]);
    const float inv = 1.f / sqrtf(turn_sum(ss, buf, turn) * inv_n + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      if (c < W) v[i] = mul4(v[i], *reinterpret_cast<const float4*>(a.w_out + c), inv);
    }
  };
  float4 before[NV];
  float* kept = nullptr;            // this CTA's state slot (it holds the sequence's first row)
  if (a.mu) {
#pragma unroll
    for (int i = 0; i < NV; ++i) before[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t0 > start) {
      float4 r[NV];
      load(t0 - 1, before, r);
      source(before, r);
      norm(before);
    } else if (a.slots[s] >= 0) {
      kept = a.state + (long long)a.slots[s] * W;
      if (a.pos[start] > 0) {
#pragma unroll
        for (int i = 0; i < NV; ++i)
          if (c0 + i * step < W) before[i] = *reinterpret_cast<const float4*>(kept + c0 + i * step);
      }
    }
  }
  constexpr bool kAhead = NV <= 4;  // the next row's loads run under this row's sums
  float4 v[NV], r[NV], v1[kAhead ? NV : 1], r1[kAhead ? NV : 1];
  if constexpr (kAhead) load(t0, v1, r1);
  for (int t = t0; t < t1; ++t) {
    if constexpr (kAhead) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        v[i] = v1[i];
        r[i] = r1[i];
      }
      if (t + 1 < t1) load(t + 1, v1, r1);
    } else {
      load(t, v, r);
    }
    source(v, r);
    const long long base = (long long)t * W;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      if (c < W) *reinterpret_cast<float4*>(a.residual_out + base + c) = v[i];
    }
    norm(v);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = c0 + i * step;
      if (c >= W) continue;
      float4 o = v[i];
      if (a.mu) {
        o = mix4(v[i], before[i], *reinterpret_cast<const float4*>(a.mu + c));
        before[i] = v[i];
      }
      st4(a.x, base + c, a.bf16, o);
    }
  }
  if (!kept) return;
  if (t1 < end) {
    load(end - 1, v, r);
    source(v, r);
    norm(v);
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (c0 + i * step < W) *reinterpret_cast<float4*>(kept + c0 + i * step) = v[i];
}

// A thread per row; the thread of a sequence's first row reads the token before it and leaves the
// sequence's last token in its place.
__global__ void __launch_bounds__(128)
bigram_rows_kernel(const int* __restrict__ ids, int* __restrict__ last, const int* __restrict__ cu,
                   const int* __restrict__ slots, const int* __restrict__ pos, int* __restrict__ out,
                   int B, int T, int one_token, long long mul_prev, long long mul_cur, int buckets) {
  US_PDL_PROLOGUE();
  const int t = blockIdx.x * 128 + threadIdx.x;
  if (t >= T) return;
  int s = t, start = t, end = t + 1;
  if (!one_token) {
    int lo = 0, hi = B - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (cu[mid] <= t) lo = mid; else hi = mid - 1;
    }
    s = lo;
    start = cu[s];
    end = cu[s + 1];
  }
  long long prev = -1;
  if (t > start) {
    prev = ids[t - 1];
  } else if (slots[s] >= 0) {
    if (pos[t] > 0) prev = last[slots[s]];
    last[slots[s]] = ids[end - 1];
  }
  out[t] = prev < 0 ? buckets : (int)((prev * mul_prev + (long long)ids[t] * mul_cur) % buckets);
}

template <int NV>
__global__ void __launch_bounds__(256)
poly_norm_kernel(const void* __restrict__ z, long long ldz, const float* __restrict__ act,
                 void* __restrict__ out, long long ldo, int W, int width, float eps, int bf16) {
  US_PDL_PROLOGUE();
  __shared__ float part[3][8];
  const int step = blockDim.x * 4, c0 = threadIdx.x * 4;
  const long long zi = (long long)blockIdx.x * ldz, oi = (long long)blockIdx.x * ldo;
  float4 v[NV];
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = c0 + i * step;
    v[i] = c < W ? ld4(z, zi + c, bf16) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float* p = reinterpret_cast<const float*>(&v[i]);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float q = p[e] * p[e];
      s2 += q;
      s4 += q * q;
      s6 += q * q * q;
    }
  }
  s2 = us::warp_sum(s2);
  s4 = us::warp_sum(s4);
  s6 = us::warp_sum(s6);
  if ((threadIdx.x & 31) == 0) {
    part[0][threadIdx.x >> 5] = s2;
    part[1][threadIdx.x >> 5] = s4;
    part[2][threadIdx.x >> 5] = s6;
  }
  __syncthreads();
  s2 = s4 = s6 = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) {
    s2 += part[0][w];
    s4 += part[1][w];
    s6 += part[2][w];
  }
  const float n = 1.f / (float)width;
  const float a = act[0] / sqrtf(s2 * n + eps), b = act[1] / sqrtf(s4 * n + eps),
              c3 = act[2] / sqrtf(s6 * n + eps), e0 = act[3];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = c0 + i * step;
    if (c >= W) continue;
    float4 o;
    const float* p = reinterpret_cast<const float*>(&v[i]);
    float* q = reinterpret_cast<float*>(&o);
#pragma unroll
    for (int e = 0; e < 4; ++e)
      q[e] = c + e < width ? fmaf(fmaf(fmaf(c3, p[e], b), p[e], a), p[e], e0) : 0.f;
    st4(out, oi + c, bf16, o);
  }
}

int block_threads(int W) { return min(256, (W / 4 + 31) / 32 * 32); }

}  // namespace

namespace {

template <int FORM, bool MIX>
int launch_stream(const StreamRows& a, cudaStream_t stream) {
  const int grid = !a.mu ? us::ceil_div(a.T, a.rows) : a.one_token ? a.T : a.T / kRows + a.B;
  const dim3 block(block_threads(a.W));
  const int nv = us::ceil_div(a.W, 1024);
#define US_STREAM(N) \
  US_CUDA_CHECK(us::launch_pdl(stream_rows_kernel<N, FORM, MIX>, dim3(grid), block, 0, stream, a))
  if (nv <= 1) US_STREAM(1);
  else if (nv <= 2) US_STREAM(2);
  else if (nv <= 4) US_STREAM(4);
  else if (nv <= 8) US_STREAM(8);
  else if (nv <= 16) US_STREAM(16);
  else return US_ERR_LIMIT;
#undef US_STREAM
  return US_OK;
}

}  // namespace

// Start of the stream (y null) or output norm and add, then the next sublayer's input rows.
US_API int us_stream_rows(const int* ids, const int* rows2, const void* table, const void* table2,
                          float scale, int vocab, int n2, const void* y, const float* residual,
                          const float* w, float* residual_out, const float* w_out, const float* mu,
                          float* state, const int* cu, const int* slots, const int* pos, void* x,
                          int B, int T, int W, int width, int bf16, int one_token, float eps,
                          void* stream_) {
  US_REQUIRE(w && residual_out && w_out && x && T >= 0 && W >= 8 && (W % 8) == 0 && width >= 1 &&
             width <= W);
  US_REQUIRE(y ? residual != nullptr && residual != residual_out : (ids && table && (!rows2 || table2)));
  US_REQUIRE(!mu || (state && cu && slots && pos && B >= 1 && (!one_token || B == T)));
  if (T == 0) return US_OK;
  StreamRows a{ids, rows2, table, table2, scale, vocab, n2, y, residual, w, residual_out, w_out, mu,
               state, cu, slots, pos, x, B, T, W, width, bf16, one_token, eps, T >= 2048 ? 4 : 1, us_status_ptr()};
  return launch_stream<kOutNorm, false>(a, (cudaStream_t)stream_);
}

// The plain form: residual_out = table row * scale (ids given), or residual + gain * (y, or the mixture
// of `top` expert rows per token); x = rms(residual_out) * w_out.
US_API int us_plain_rows(const int* ids, const void* table, float scale, int vocab, const void* y,
                         const void* y_perm, const int* perm, const float* route_w, int top,
                         const void* ident, const void* shared, float gain, const float* residual,
                         float* residual_out, const float* w_out, void* x, int T, int W, int width,
                         int bf16, float eps, void* stream_) {
  US_REQUIRE(residual_out && w_out && x && T >= 0 && W >= 8 && (W % 8) == 0 && width >= 1 && width <= W);
  US_REQUIRE(y || y_perm ? residual && residual != residual_out : ids && table);
  US_REQUIRE(!y_perm || (perm && route_w && top >= 1 && top <= 32 && !y));
  if (T == 0) return US_OK;
  StreamRows a{ids, nullptr, table, nullptr, scale, vocab, 0, y, residual, nullptr, residual_out, w_out, nullptr,
               nullptr, nullptr, nullptr, nullptr, x, 1, T, W, width, bf16, 0, eps, T >= 2048 ? 2 : 1, us_status_ptr(),
               y || y_perm ? gain : 1.f, y_perm, perm, route_w, top, ident, shared};
  return y_perm ? launch_stream<kPlain, true>(a, (cudaStream_t)stream_) : launch_stream<kPlain, false>(a, (cudaStream_t)stream_);
}

// The layer form: residual_out = table row * scale (ids given), or residual + ln(y, or a mixture of `top`
// expert rows per token and a shared row) * w + b; x = residual_out, or with w_out its layer norm.
US_API int us_layer_rows(const int* ids, const void* table, float scale, int vocab, const void* y,
                         const void* y_perm, const int* perm, const float* route_w, int top,
                         const void* shared, const float* shared_gate, long long ld_gate,
                         const float* residual, const float* w, const float* b, float* residual_out,
                         const float* w_out, const float* b_out, void* x, int T, int W, int width,
                         int bf16, float eps, void* stream_) {
  US_REQUIRE(residual_out && x && T >= 0 && W >= 8 && (W % 8) == 0 && width >= 1 && width <= W);
  US_REQUIRE(y || y_perm ? residual && residual != residual_out && w && b : ids && table && !residual);
  US_REQUIRE(!y_perm || (perm && route_w && top >= 1 && top <= 32 && !y));
  US_REQUIRE(!w_out || b_out);
  if (T == 0) return US_OK;
  StreamRows a{ids, nullptr, table, nullptr, scale, vocab, 0, y, residual, w, residual_out, w_out, nullptr,
               nullptr, nullptr, nullptr, nullptr, x, 1, T, W, width, bf16, 0, eps, T >= 2048 ? 2 : 1, us_status_ptr(),
               1.f, y_perm, perm, route_w, top, nullptr, shared, b, b_out, shared_gate, ld_gate};
  return y_perm ? launch_stream<kLayer, true>(a, (cudaStream_t)stream_) : launch_stream<kLayer, false>(a, (cudaStream_t)stream_);
}

US_API int us_bigram_rows(const int* ids, int* last, const int* cu, const int* slots, const int* pos,
                          int* out, int B, int T, int one_token, long long mul_prev,
                          long long mul_cur, int buckets, void* stream_) {
  US_REQUIRE(ids && last && cu && slots && pos && out && B >= 1 && T >= 0 && buckets >= 1);
  US_REQUIRE(!one_token || B == T);
  if (T == 0) return US_OK;
  US_CUDA_CHECK(us::launch_pdl(bigram_rows_kernel, dim3((T + 127) / 128), dim3(128), 0,
                               (cudaStream_t)stream_, ids, last, cu, slots, pos, out, B, T, one_token,
                               mul_prev, mul_cur, buckets));
  return US_OK;
}

US_API int us_poly_norm(const void* z, long long ldz, const float* act, void* out, long long ldo,
                        int T, int W, int width, float eps, int bf16, void* stream_) {
  US_REQUIRE(z && act && out && T >= 0 && W >= 4 && (W % 4) == 0 && width >= 1 && width <= W &&
             (ldz % 4) == 0 && (ldo % 4) == 0);
  if (T == 0) return US_OK;
  const dim3 block(block_threads(W));
  const int nv = us::ceil_div(W, 1024);
#define US_POLY(N)                                                                                \
  US_CUDA_CHECK(us::launch_pdl(poly_norm_kernel<N>, dim3(T), block, 0, (cudaStream_t)stream_, z, ldz, \
                               act, out, ldo, W, width, eps, bf16))
  if (nv <= 1) US_POLY(1);
  else if (nv <= 2) US_POLY(2);
  else if (nv <= 4) US_POLY(4);
  else if (nv <= 8) US_POLY(8);
  else if (nv <= 16) US_POLY(16);
  else return US_ERR_LIMIT;
#undef US_POLY
  return US_OK;
}
