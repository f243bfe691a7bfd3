// Softmax attention with grouped heads over cache pages, for layers whose queries and keys are normed
// per head and turned by position, whose window slides and whose softmax has a sink:
//
//   s_h(i, j) = scale q_h(i) . k_g(j),   j <= i, i - j < window (0: no limit),   g = h / (H / G)
//   o_h(i)    = sum_j e^{s_h(i, j)} v_g(j) / (sum_j e^{s_h(i, j)} + e^{sink_h})
//
// or, with weights that do not depend on the other keys (a temperature and a shift per head, capped scores),
//
//   w_h(i, j) = sigmoid(cap tanh(temp_h s_h(i, j) / cap) + shift_h),   o_h(i) = sum_j w_h(i, j) v_g(j)
//
//   us_window_prep             RMS norm over each head, rotation of its first channels, q into rows of
//                              their own, k and v into pages
//   us_window_gather           the keys and values that a batch's prompts see, from pages into packed rows
//   us_window_attention_rows   any sizes, bf16 or FP32: one CTA per (query row, key head)
//
// (prompts: us_window_flash; single rows: us_paged_decode_attention_sink, us_sigmoid_decode).  Channel i
// turns with channel i + n, n the number of pairs, or 2i with 2i + 1 (neighbours).  The angle is formed and reduced to a fraction of a turn in FP64, so
// far positions lose nothing before the FP32 sine and cosine.
#include "include/us_common.cuh"

namespace {

__device__ __forceinline__ float ld1(const void* base, long long i, int bf16) {
  return bf16 ? us::bf2f(reinterpret_cast<const __nv_bfloat16*>(base)[i])
              : reinterpret_cast<const float*>(base)[i];
}
__device__ __forceinline__ void st1(void* base, long long i, int bf16, float v) {
  if (bf16) reinterpret_cast<__nv_bfloat16*>(base)[i] = us::f2bf(v);
  else reinterpret_cast<float*>(base)[i] = v;
}
// VEC neighbouring elements (2: i even)
template <int VEC>
__device__ __forceinline__ void ldv(float (&o)[VEC], const void* base, long long i, int bf16) {
  if (VEC == 2 && bf16) {
    const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(reinterpret_cast<const __nv_bfloat16*>(base) + i);
    o[0] = us::bf2f(v.x);
    o[VEC - 1] = us::bf2f(v.y);
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = ld1(base, i + e, bf16);
  }
}
template <int VEC>
__device__ __forceinline__ void stv(void* base, long long i, int bf16, const float (&v)[VEC]) {
  if (VEC == 2 && bf16) {
    *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<__nv_bfloat16*>(base) + i) =
        __floats2bfloat162_rn(v[0], v[VEC - 1]);
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) st1(base, i + e, bf16, v[e]);
  }
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

// ------------------------------------------------------------- preparation --
constexpr int kPrepWarps = 4, kPrepHeads = 4;

struct Prep {
  const void* x;                // projection rows: q heads from off_q, k heads from off_k, v heads from off_v
  long long ldx;
  int off_q, off_k, off_v, H, G, D, V, pairs;
  const float *wq, *wk;         // [D]
  const double* freq;           // [pairs]
  float mag;                    // factor on cosine and sine
  const int *pos, *slots;
  void* q;                      // [T, H, Dq], columns D .. Dq zero
  int Dq;
  void *kp, *vp;                // pages [n, page, G, D], [n, page, G, V]
  int T, bf16;
  float eps;
  int neighbours;
};

// A warp takes up to kPrepHeads heads of one token, whose sines and cosines it forms once.  A lane holds
// VEC neighbouring channels out of every 32 VEC; the rotation's partners meet in shared memory.
template <int NI, int VEC>
__global__ void __launch_bounds__(kPrepWarps * 32) window_prep_kernel(const Prep a) {
  US_PDL_PROLOGUE();
  __shared__ float buf[kPrepWarps][NI * 32 * VEC];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* sm = buf[warp];
  const int units = a.H + a.G, groups = (units + kPrepHeads - 1) / kPrepHeads;
  const long long item = (long long)blockIdx.x * kPrepWarps + warp;
  if (item >= (long long)a.T * groups) return;
  const int t = (int)(item / groups), u0 = (int)(item % groups) * kPrepHeads;
  const int n = a.pairs, pos = a.pos[t];
  const long long slot = a.slots[t];
  float cs[NI][VEC], sn[NI][VEC];
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      const int p = (i * 32 + lane) * VEC + e;
      if (p < n) {
        turn(pos, a.freq[p], cs[i][e], sn[i][e]);
        cs[i][e] *= a.mag;
        sn[i][e] *= a.mag;
      }
    }
  for (int unit = u0; unit < min(units, u0 + kPrepHeads); ++unit) {
    const bool is_q = unit < a.H;
    const int g = unit - a.H;
    if (!is_q && slot < 0) break;
    const long long from = (long long)t * a.ldx + (is_q ? a.off_q + unit * a.D : a.off_k + g * a.D);
    const float* w = is_q ? a.wq : a.wk;
    float v[NI][VEC], ss = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = (i * 32 + lane) * VEC;
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[i][e] = 0.f;
      if (d < a.D) ldv<VEC>(v[i], a.x, from + d, a.bf16);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += v[i][e] * v[i][e];
    }
    const float inv = 1.f / sqrtf(us::warp_sum(ss) / (float)a.D + a.eps);
    void* dst = is_q ? a.q : a.kp;
    const long long to = is_q ? ((long long)t * a.H + unit) * a.Dq : (slot * a.G + g) * a.D;
    __syncwarp();
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = (i * 32 + lane) * VEC;
      if (d >= a.D) continue;
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        v[i][e] *= inv * w[d + e];
        sm[d + e] = v[i][e];
      }
      if (d >= 2 * n) stv<VEC>(dst, to + d, a.bf16, v[i]);
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int p = (i * 32 + lane) * VEC;
      if (p >= n) continue;
      float lo[VEC], hi[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const float x = a.neighbours ? sm[2 * (p + e)] : sm[p + e];
        const float y = a.neighbours ? sm[2 * (p + e) + 1] : sm[p + n + e];
        lo[e] = x * cs[i][e] - y * sn[i][e];
        hi[e] = y * cs[i][e] + x * sn[i][e];
      }
      if (!a.neighbours) {
        stv<VEC>(dst, to + p, a.bf16, lo);
        stv<VEC>(dst, to + p + n, a.bf16, hi);
      } else if constexpr (VEC == 2) {
        const float first[VEC] = {lo[0], hi[0]}, second[VEC] = {lo[VEC - 1], hi[VEC - 1]};
        stv<VEC>(dst, to + 2 * p, a.bf16, first);
        stv<VEC>(dst, to + 2 * p + 2, a.bf16, second);
      } else {
        st1(dst, to + 2 * p, a.bf16, lo[0]);
        st1(dst, to + 2 * p + 1, a.bf16, hi[0]);
      }
    }
    if (is_q) {
      for (int d = a.D + lane; d < a.Dq; d += 32) st1(dst, to + d, a.bf16, 0.f);
    } else {
      const long long vf = (long long)t * a.ldx + a.off_v + (long long)g * a.V, vt = (slot * a.G + g) * a.V;
      for (int d = lane * VEC; d < a.V; d += 32 * VEC) {
        float x[VEC];
        ldv<VEC>(x, a.x, vf + d, a.bf16);
        stv<VEC>(a.vp, vt + d, a.bf16, x);
      }
    }
  }
}

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

// The same for neighbouring channels: a lane holds both of every pair, four channels at a time, and a
// warp's heads are loaded together.
template <int NI>
__global__ void __launch_bounds__(kPrepWarps * 32) neighbours_prep_kernel(const Prep a) {
  US_PDL_PROLOGUE();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int units = a.H + a.G, groups = (units + kPrepHeads - 1) / kPrepHeads;
  const long long item = (long long)blockIdx.x * kPrepWarps + warp;
  if (item >= (long long)a.T * groups) return;
  const int t = (int)(item / groups), u0 = (int)(item % groups) * kPrepHeads, pos = a.pos[t];
  const long long slot = a.slots[t], row = (long long)t * a.ldx;
  float4 v[kPrepHeads][NI];
  bool in[kPrepHeads];
#pragma unroll
  for (int u = 0; u < kPrepHeads; ++u) {
    const int unit = u0 + u;
    in[u] = unit < a.H || (unit < units && slot >= 0);
    const long long from = row + (unit < a.H ? a.off_q + unit * a.D : a.off_k + (unit - a.H) * a.D);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = (i * 32 + lane) * 4;
      v[u][i] = in[u] && d < a.D ? ld4(a.x, from + d, a.bf16) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  float cs[NI][2], sn[NI][2];
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int p = (i * 32 + lane) * 2 + e;
      cs[i][e] = 1.f;
      sn[i][e] = 0.f;
      if (p < a.pairs) {
        turn(pos, a.freq[p], cs[i][e], sn[i][e]);
        cs[i][e] *= a.mag;
        sn[i][e] *= a.mag;
      }
    }
  float ss[kPrepHeads];
#pragma unroll
  for (int u = 0; u < kPrepHeads; ++u) {
    ss[u] = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i)
      ss[u] += v[u][i].x * v[u][i].x + v[u][i].y * v[u][i].y + v[u][i].z * v[u][i].z + v[u][i].w * v[u][i].w;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int u = 0; u < kPrepHeads; ++u) ss[u] += __shfl_xor_sync(0xffffffffu, ss[u], o);
#pragma unroll
  for (int u = 0; u < kPrepHeads; ++u) {
    const int unit = u0 + u, g = unit - a.H;
    if (!in[u]) continue;
    const bool is_q = g < 0;
    const float* w = is_q ? a.wq : a.wk;
    void* dst = is_q ? a.q : a.kp;
    const long long to = is_q ? ((long long)t * a.H + unit) * a.Dq : (slot * a.G + g) * a.D;
    const float inv = 1.f / sqrtf(ss[u] / (float)a.D + a.eps);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int d = (i * 32 + lane) * 4;
      if (d < a.D) {
        const float4 w4 = *reinterpret_cast<const float4*>(w + d);
        const float4 n = make_float4(v[u][i].x * (inv * w4.x), v[u][i].y * (inv * w4.y), v[u][i].z * (inv * w4.z),
                                     v[u][i].w * (inv * w4.w));
        st4(dst, to + d, a.bf16, make_float4(n.x * cs[i][0] - n.y * sn[i][0], n.y * cs[i][0] + n.x * sn[i][0],
                                             n.z * cs[i][1] - n.w * sn[i][1], n.w * cs[i][1] + n.z * sn[i][1]));
      } else if (is_q && d < a.Dq) {
        st4(dst, to + d, a.bf16, make_float4(0.f, 0.f, 0.f, 0.f));
      }
    }
    if (is_q) continue;
    const long long vf = row + a.off_v + (long long)g * a.V, vt = (slot * a.G + g) * a.V;
    for (int d = lane * 4; d < a.V; d += 128) st4(a.vp, vt + d, a.bf16, ld4(a.x, vf + d, a.bf16));
  }
}

template <int VEC>
int launch_prep(const Prep& a, cudaStream_t stream) {
  const long long items = (long long)a.T * ((a.H + a.G + kPrepHeads - 1) / kPrepHeads);
  const dim3 grid((unsigned)((items + kPrepWarps - 1) / kPrepWarps)), block(kPrepWarps * 32);
  const int ni = us::ceil_div(a.D, 32 * VEC);
  if (ni <= 1) US_CUDA_CHECK(us::launch_pdl(window_prep_kernel<1, VEC>, grid, block, 0, stream, a));
  else if (ni <= 2) US_CUDA_CHECK(us::launch_pdl(window_prep_kernel<2, VEC>, grid, block, 0, stream, a));
  else if (ni <= 4) US_CUDA_CHECK(us::launch_pdl(window_prep_kernel<4, VEC>, grid, block, 0, stream, a));
  else if (ni <= 8) US_CUDA_CHECK(us::launch_pdl(window_prep_kernel<8, VEC>, grid, block, 0, stream, a));
  else if (ni <= 16) US_CUDA_CHECK(us::launch_pdl(window_prep_kernel<16, VEC>, grid, block, 0, stream, a));
  else return US_ERR_LIMIT;
  return US_OK;
}

// ------------------------------------------------------------------ gather --
struct Gather {
  const __nv_bfloat16 *kp, *vp;          // pages [n, page, G, D], [n, page, G, V]
  int G, D, V, Dp, Vp, page, max_pages;
  __nv_bfloat16 *k, *v;                  // [rows, G, Dp], [rows, G, Vp], zero past D and V
  int* cu_k;                             // [B + 1]
  const int *cu, *pos, *page_table;
  int B, window, min_rows, rows;
};

// keys that sequence s sees in this batch (0: too few rows, it is served elsewhere) and the first one
__device__ __forceinline__ int seen(const Gather& a, int s, int& first) {
  const int q = a.cu[s + 1] - a.cu[s];
  first = 0;
  if (q < a.min_rows) return 0;
  const int p0 = a.pos[a.cu[s]];
  first = a.window > 0 ? max(0, p0 - a.window + 1) : 0;
  return p0 + q - first;
}

template <bool WIDE>
__device__ __forceinline__ void copy_heads(__nv_bfloat16* to, const __nv_bfloat16* from, int G, int D, int Dp) {
  const int lane = threadIdx.x & 31;
  if (WIDE) {
    const int per = Dp / 8;
    for (int e = lane; e < G * per; e += 32) {
      const int g = e / per, c = (e - g * per) * 8;
      *reinterpret_cast<uint4*>(to + (long long)e * 8) =
          c < D ? *reinterpret_cast<const uint4*>(from + g * D + c) : make_uint4(0, 0, 0, 0);
    }
  } else {
    for (int e = lane; e < G * Dp; e += 32) {
      const int g = e / Dp, c = e - g * Dp;
      to[e] = c < D ? from[g * D + c] : us::f2bf(0.f);
    }
  }
}

// A warp per key row; the first thread also writes the sequences' offsets.
template <bool WIDE>
__global__ void __launch_bounds__(256) window_gather_kernel(const Gather a) {
  US_PDL_PROLOGUE();
  int at = 0, first = 0;
  if (blockIdx.x == 0 && threadIdx.x == 0) {
    for (int s = 0; s < a.B; ++s) {
      a.cu_k[s] = at;
      at += seen(a, s, first);
    }
    a.cu_k[a.B] = at;
  }
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (row >= a.rows) return;
  at = 0;
  for (int s = 0; s < a.B; ++s) {
    const int n = seen(a, s, first);
    if (row < at + n) {
      const int key = first + row - at;
      const long long src =
          (long long)a.page_table[(long long)s * a.max_pages + key / a.page] * a.page + key % a.page;
      copy_heads<WIDE>(a.k + (long long)row * a.G * a.Dp, a.kp + src * a.G * a.D, a.G, a.D, a.Dp);
      copy_heads<WIDE>(a.v + (long long)row * a.G * a.Vp, a.vp + src * a.G * a.V, a.G, a.V, a.Vp);
      return;
    }
    at += n;
  }
}

// ---------------------------------------------------------------- row form --
struct RowAttn {
  const void* q;              // [T, H, D]: rows at ldq, heads at hsq
  long long ldq;
  int hsq;
  const void *kp, *vp;        // pages [n, page, G, D], [n, page, G, V]
  void* out;                  // [T, ldo], head h at column h V
  long long ldo;
  const int *cu, *pos, *seq_lens, *page_table;
  const float* sink;          // [H] or null
  int B, H, G, D, V, page, max_pages, window, bf16, per;
  float scale, out_scale;
  const float *temp, *shift;  // [H]: sigmoid weights, or null: softmax
  float cap;                  // 0: none
  const void* gate;           // head h's output times sigmoid(gate[t * ldg + h]), or null
  long long ldg;
};

constexpr int kRowThreads = 256;
constexpr int kRowKeys = 32;

// `per` query heads of one key head at a time.
__global__ void __launch_bounds__(kRowThreads) window_rows_kernel(const RowAttn a) {
  US_PDL_PROLOGUE();
  extern __shared__ __align__(16) float smf[];
  const int D = a.D, V = a.V, ldk = D | 1, rep = a.H / a.G;
  float* qs = smf;                         // [per][D], scaled
  float* ks = qs + a.per * D;              // [kRowKeys][ldk]
  float* vs = ks + kRowKeys * ldk;         // [kRowKeys][V]
  float* os = vs + kRowKeys * V;           // [per][V]
  float* ps = os + a.per * V;              // [per][kRowKeys]
  float* mx = ps + a.per * kRowKeys;       // [per] each
  float* sum = mx + a.per;
  float* fac = sum + a.per;
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int parts = (rep + a.per - 1) / a.per, g = blockIdx.y / parts, part = blockIdx.y - g * parts;
  const int h0 = g * rep + part * a.per, nh = min(a.per, rep - part * a.per);
  const int s = seq_of(a.cu, a.B, t);
  const bool live = !a.seq_lens || a.seq_lens[s] > 0;
  for (int e = tid; e < nh * D; e += kRowThreads) {
    const int h = e / D, d = e - h * D;
    qs[e] = live ? ld1(a.q, t * a.ldq + (long long)(h0 + h) * a.hsq + d, a.bf16) * a.scale : 0.f;
  }
  for (int e = tid; e < nh; e += kRowThreads) { mx[e] = -INFINITY; sum[e] = 0.f; }
  for (int e = tid; e < nh * V; e += kRowThreads) os[e] = 0.f;
  const int i = live ? a.pos[t] : -1;
  const int lo = a.window > 0 ? max(0, i - a.window + 1) : 0;
  const int* pt = a.page_table + (long long)s * a.max_pages;
  for (int j0 = lo; j0 <= i; j0 += kRowKeys) {
    const int nj = min(kRowKeys, i - j0 + 1);
    __syncthreads();
    for (int e = tid; e < nj * (D + V); e += kRowThreads) {
      const int j = e / (D + V), d = e - j * (D + V), key = j0 + j;
      const long long at = ((long long)pt[key / a.page] * a.page + key % a.page) * a.G + g;
      if (d < D) ks[j * ldk + d] = ld1(a.kp, at * D + d, a.bf16);
      else vs[j * V + d - D] = ld1(a.vp, at * V + d - D, a.bf16);
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
      float sc = ps[h * kRowKeys + lane];
      if (a.shift) {
        if (lane < nj) {
          sc *= a.temp[h0 + h];
          if (a.cap > 0.f) sc = a.cap * tanhf(sc / a.cap);
          sc = 1.f / (1.f + expf(-(sc + a.shift[h0 + h])));
        }
        ps[h * kRowKeys + lane] = lane < nj ? sc : 0.f;
        if (lane == 0) fac[h] = 1.f;
        continue;
      }
      const float m0 = mx[h], m = fmaxf(m0, us::warp_max(sc));
      const float p = lane < nj ? expf(sc - m) : 0.f;
      const float add = us::warp_sum(p);
      ps[h * kRowKeys + lane] = p;
      __syncwarp();
      if (lane == 0) {
        fac[h] = expf(m0 - m);
        sum[h] = sum[h] * fac[h] + add;
        mx[h] = m;
      }
    }
    __syncthreads();
    for (int e = tid; e < nh * V; e += kRowThreads) {
      const int h = e / V, c = e - h * V;
      float acc = os[e] * fac[h];
      for (int j = 0; j < nj; ++j) acc = fmaf(ps[h * kRowKeys + j], vs[j * V + c], acc);
      os[e] = acc;
    }
  }
  __syncthreads();
  for (int e = tid; e < nh * V; e += kRowThreads) {
    const int h = e / V, c = e - h * V;
    const float den = live && !a.shift ? sum[h] + (a.sink ? expf(a.sink[h0 + h] - mx[h]) : 0.f) : 1.f;
    float o = live ? a.out_scale * os[e] / den : 0.f;
    if (a.gate) o /= 1.f + expf(-ld1(a.gate, t * a.ldg + h0 + h, a.bf16));
    st1(a.out, t * a.ldo + (long long)(h0 + h) * V + c, a.bf16, o);
  }
}

bool even(long long a, long long b, long long c, long long d) { return ((a | b | c | d) & 1) == 0; }

}  // namespace

// v heads start at column off_v (off_k: the values are the keys as projected).  Rows with a negative slot
// write no page.
US_API int us_window_prep(const void* x, long long ldx, int off_q, int off_k, int off_v, int H, int G,
                          int D, int V, const float* wq, const float* wk, const double* freq, int pairs,
                          float mag, const int* pos, const int* slots, void* q, int Dq, void* kpages,
                          void* vpages, int T, float eps, int neighbours, int bf16, void* stream_) {
  US_REQUIRE(x && wq && wk && pos && slots && q && kpages && vpages && T >= 0 && H >= 1 && G >= 1 &&
             D >= 1 && V >= 1 && Dq >= D && 2 * pairs <= D && (pairs == 0 || freq));
  if (T == 0) return US_OK;
  Prep a{x, ldx, off_q, off_k, off_v, H, G, D, V, pairs, wq, wk, freq, mag, pos, slots, q, Dq, kpages, vpages,
         T, bf16, eps, neighbours};
  const int sizes = D | V | Dq | off_q | off_k | off_v | (int)(ldx & 3);
  if (neighbours && (sizes & 3) == 0 && D <= 256 && Dq <= 128 * us::ceil_div(D, 128) && ((uintptr_t)x % 16) == 0 &&
      ((uintptr_t)wq % 16) == 0 && ((uintptr_t)wk % 16) == 0) {
    const long long items = (long long)T * ((H + G + kPrepHeads - 1) / kPrepHeads);
    const dim3 grid((unsigned)((items + kPrepWarps - 1) / kPrepWarps)), block(kPrepWarps * 32);
    US_CUDA_CHECK(us::launch_pdl(D <= 128 ? neighbours_prep_kernel<1> : neighbours_prep_kernel<2>, grid, block, 0,
                                 (cudaStream_t)stream_, a));
    return US_OK;
  }
  const bool two = even(ldx, off_q, off_k, off_v) && even(D, V, pairs, Dq) && ((uintptr_t)x % 4) == 0;
  return two ? launch_prep<2>(a, (cudaStream_t)stream_) : launch_prep<1>(a, (cudaStream_t)stream_);
}

// Packs what sequences of at least `min_rows` rows see (window 0: everything) into k [rows, G, Dp] and
// v [rows, G, Vp]; writes their offsets to cu_k.  `rows` is their number, known to the host.
US_API int us_window_gather(const void* kpages, const void* vpages, int G, int D, int V, int Dp, int Vp,
                            void* k, void* v, int* cu_k, const int* cu, const int* pos,
                            const int* page_table, int B, int page, int max_pages, int window,
                            int min_rows, int rows, void* stream_) {
  US_REQUIRE(kpages && vpages && k && v && cu_k && cu && pos && page_table && B >= 1 && page >= 1 &&
             rows >= 1 && min_rows >= 1 && G >= 1 && Dp >= D && Vp >= V && (Dp % 8) == 0 && (Vp % 8) == 0);
  Gather a{(const __nv_bfloat16*)kpages, (const __nv_bfloat16*)vpages, G, D, V, Dp, Vp, page, max_pages,
           (__nv_bfloat16*)k, (__nv_bfloat16*)v, cu_k, cu, pos, page_table, B, window, min_rows, rows};
  const dim3 grid(us::ceil_div(rows, 8)), block(256);
  cudaStream_t stream = (cudaStream_t)stream_;
  if (((D | V) % 8) == 0) US_CUDA_CHECK(us::launch_pdl(window_gather_kernel<true>, grid, block, 0, stream, a));
  else US_CUDA_CHECK(us::launch_pdl(window_gather_kernel<false>, grid, block, 0, stream, a));
  return US_OK;
}

// Attention of T rows (rows of sequence s at cu[s] .. cu[s + 1], keys up to a row's own position).  seq_lens
// [B] or null: length 0 marks padding, whose rows become zero.  temp and shift [H] (both or none): sigmoid
// weights with scores capped at `cap` (0: not).  gate (or null): a logit per row and head.
US_API int us_window_attention_rows(const void* q, long long ldq, int hsq, const void* kpages,
                                    const void* vpages, void* out, long long ldo, const int* cu,
                                    const int* pos, const int* seq_lens, const int* page_table,
                                    const float* sink, int T, int B, int H, int G, int D, int V, int page,
                                    int max_pages, int window, float scale, float out_scale,
                                    const float* temp, const float* shift, float cap, const void* gate,
                                    long long ldg, int bf16, void* stream_) {
  US_REQUIRE(q && kpages && vpages && out && cu && pos && page_table && T >= 0 && B >= 1 && H >= 1 &&
             G >= 1 && H % G == 0 && D >= 1 && V >= 1 && page >= 1 && ldo >= (long long)H * V && !temp == !shift);
  if (T == 0) return US_OK;
  constexpr size_t kMost = 220 * 1024;
  auto bytes = [&](int per) {
    return 4 * ((size_t)per * (D + V + kRowKeys + 3) + (size_t)kRowKeys * ((D | 1) + V));
  };
  const int rep = H / G;
  int per = rep < 16 ? rep : 16;
  while (per > 1 && bytes(per) > kMost) per /= 2;
  const int parts = us::ceil_div(rep, per);
  if (bytes(per) > kMost || (long long)G * parts > 65535) return US_ERR_LIMIT;
  RowAttn a{q, ldq, hsq, kpages, vpages, out, ldo, cu, pos, seq_lens, page_table, sink, B, H, G, D, V, page,
            max_pages, window, bf16, per, scale, out_scale, temp, shift, cap, gate, ldg};
  static bool configured = false;
  if (!configured) {
    US_CUDA_CHECK(cudaFuncSetAttribute(window_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMost));
    configured = true;
  }
  US_CUDA_CHECK(us::launch_pdl(window_rows_kernel, dim3(T, G * parts), dim3(kRowThreads), bytes(per),
                               (cudaStream_t)stream_, a));
  return US_OK;
}
