// Recurrent token mixers over a ragged step: each layer carries a matrix state S [key dimension, value dimension] per head and
// sequence, in fp32, in a slot of the state pool.  The rows of a step are the new tokens of several requests; entry e continues
// the slot entry_slot[e] (from zero when entry_ctx[e] == 0) and leaves its new state there.
//
//   pg_short_conv        causal convolution over time per channel (+ bias), silu; the last taps - 1 inputs of a sequence live in an
//                        fp32 slot; optionally the inverse Euclidean norm of every group of channels (a head's vector) of a row
//   pg_delta_scan        delta rule with one decay per head and KEY CHANNEL: S <- g * S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q
//   pg_gated_scan        S <- a S + w k v^T, o = S^T q with one scalar decay a and write weight w per head and token, in two forms:
//                        state space (a = exp(-r dt), w = dt, plus a skip D v) and exponentially gated matrix memory (running maximum,
//                        normaliser vector)
//   pg_group_norm_gate   per-group RMS norm of the read-out with an output gate before or after it
//
// Scans step token by token (decoded tokens, short portions, any head size, both activation types); the block forms of the same
// recurrences for prompt portions are in seq_recurrence_mma.cu.
#include "common.cuh"
#include "paligemma_b200.h"

using bf16 = __nv_bfloat16;

#define PG_ST(s) reinterpret_cast<cudaStream_t>(s)
#define PG_RET()                                                    \
  do {                                                              \
    pg_count_launch(1);                                             \
    return cudaGetLastError() == cudaSuccess ? PG_OK : PG_ERR_CUDA; \
  } while (0)

namespace {

__device__ __forceinline__ float ld(const float* p, long long i) { return p[i]; }
__device__ __forceinline__ float ld(const bf16* p, long long i) { return __bfloat162float(p[i]); }
__device__ __forceinline__ void st(float* p, long long i, float v) { p[i] = v; }
__device__ __forceinline__ void st(bf16* p, long long i, float v) { p[i] = __float2bfloat16_rn(v); }

template <int V>
__device__ __forceinline__ void ldv(const float* p, long long i, float* v) {
#pragma unroll
  for (int k = 0; k < V; ++k) v[k] = p[i + k];
}
template <>
__device__ __forceinline__ void ldv<4>(const float* p, long long i, float* v) {
  const float4 a = *reinterpret_cast<const float4*>(p + i);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
template <>
__device__ __forceinline__ void ldv<2>(const float* p, long long i, float* v) {
  const float2 a = *reinterpret_cast<const float2*>(p + i);
  v[0] = a.x; v[1] = a.y;
}
template <int V>
__device__ __forceinline__ void ldv(const bf16* p, long long i, float* v) {
#pragma unroll
  for (int k = 0; k < V; ++k) v[k] = __bfloat162float(p[i + k]);
}
template <>
__device__ __forceinline__ void ldv<4>(const bf16* p, long long i, float* v) {
  const uint2 u = *reinterpret_cast<const uint2*>(p + i);
  v[0] = __uint_as_float(u.x << 16); v[1] = __uint_as_float(u.x & 0xffff0000u);
  v[2] = __uint_as_float(u.y << 16); v[3] = __uint_as_float(u.y & 0xffff0000u);
}
template <>
__device__ __forceinline__ void ldv<2>(const bf16* p, long long i, float* v) {
  const uint32_t u = *reinterpret_cast<const uint32_t*>(p + i);
  v[0] = __uint_as_float(u << 16); v[1] = __uint_as_float(u & 0xffff0000u);
}
template <int V>
__device__ __forceinline__ void stv(float* p, long long i, const float* v) {
#pragma unroll
  for (int k = 0; k < V; ++k) p[i + k] = v[k];
}
template <>
__device__ __forceinline__ void stv<4>(float* p, long long i, const float* v) { *reinterpret_cast<float4*>(p + i) = make_float4(v[0], v[1], v[2], v[3]); }
template <>
__device__ __forceinline__ void stv<2>(float* p, long long i, const float* v) { *reinterpret_cast<float2*>(p + i) = make_float2(v[0], v[1]); }
template <int V>
__device__ __forceinline__ void stv(bf16* p, long long i, const float* v) {
#pragma unroll
  for (int k = 0; k < V; ++k) p[i + k] = __float2bfloat16_rn(v[k]);
}
template <>
__device__ __forceinline__ void stv<2>(bf16* p, long long i, const float* v) { *reinterpret_cast<uint32_t*>(p + i) = pg::pack_bf16(v[0], v[1]); }
template <>
__device__ __forceinline__ void stv<4>(bf16* p, long long i, const float* v) {
  *reinterpret_cast<uint2*>(p + i) = make_uint2(pg::pack_bf16(v[0], v[1]), pg::pack_bf16(v[2], v[3]));
}

__device__ __forceinline__ float wsum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ---------------------------------------------------------------------------------------------------------------------
// Short convolution.  Channels come in groups (a head's vector; groups of a section without a norm are arbitrary runs of
// channels); one warp walks a run of `chunk` consecutive rows of one entry for one group, lane <-> V adjacent channels x NK, the last
// taps - 1 inputs in registers.  Only the warp of an entry's FIRST run reads the slot, and that warp alone writes it (the entry's
// last inputs, re-read from x), so no other warp of the launch touches it; chunk >= taps - 1 by construction.
// ---------------------------------------------------------------------------------------------------------------------
template <typename TA, int V, int NK, int TAPS>
__global__ void __launch_bounds__(128) short_conv_kernel(const TA* __restrict__ x, long long ldx, const float* __restrict__ w,
                                                         const float* __restrict__ bias, float* __restrict__ state, TA* __restrict__ out,
                                                         long long ldo, float* __restrict__ inv, int ldi, PgConvSections sec, int taps, int C,
                                                         const int* __restrict__ entry_row0, const int* __restrict__ entry_n,
                                                         const int* __restrict__ entry_ctx, const int* __restrict__ entry_slot, int chunk) {
  const int e = blockIdx.z, lane = threadIdx.x & 31;
  const int n = entry_n[e], r0 = blockIdx.y * chunk;
  if (r0 >= n) return;
  int g = blockIdx.x * 4 + (threadIdx.x >> 5), s = 0, unit_base = 0;
  while (s < sec.count && g >= sec.groups[s]) {
    g -= sec.groups[s];
    if (sec.unit[s]) unit_base += sec.groups[s];
    ++s;
  }
  if (s >= sec.count) return;
  const int size = sec.size[s], width = min(size, sec.total[s] - g * size);  // the last group of a section without a norm may be short
  const long long row0 = entry_row0[e];
  const long long xc = sec.xcol[s] + (long long)g * size, cc = sec.ccol[s] + (long long)g * size;
  const int K = taps - 1;
  float* slot = state + (long long)entry_slot[e] * K * C + cc;
  float wt[TAPS][NK * V], bs[NK * V], hist[TAPS - 1 > 0 ? TAPS - 1 : 1][NK * V];
  // tap j of the kernel is `TAPS - 1 - j` tokens back; unused older taps carry zero weights
#pragma unroll
  for (int k = 0; k < NK; ++k) {
    const int c = k * 32 * V + lane * V;
#pragma unroll
    for (int v = 0; v < V; ++v) {
      const bool ok = c + v < width;
      bs[k * V + v] = (bias != nullptr && ok) ? bias[cc + c + v] : 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const int tj = j - (TAPS - taps);
        wt[j][k * V + v] = (ok && tj >= 0) ? w[(long long)tj * C + cc + c + v] : 0.f;
      }
      // hist[j] = input of row r0 - (TAPS - 1) + j
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int row = r0 - (TAPS - 1) + j;
        float h = 0.f;
        if (ok) {
          if (row >= 0) h = ld(x, (row0 + row) * ldx + xc + c + v);
          else if (entry_ctx[e] > 0 && K + row >= 0) h = slot[(long long)(K + row) * C + c + v];
        }
        hist[j][k * V + v] = h;
      }
    }
  }
  const int r1 = min(n, r0 + chunk);
  for (int r = r0; r < r1; ++r) {
    float ss = 0.f, y[NK * V];
#pragma unroll
    for (int k = 0; k < NK; ++k) {
      const int c = k * 32 * V + lane * V;
      float cur[V];
      if (c + V <= width) ldv<V>(x, (row0 + r) * ldx + xc + c, cur);
      else {
#pragma unroll
        for (int v = 0; v < V; ++v) cur[v] = c + v < width ? ld(x, (row0 + r) * ldx + xc + c + v) : 0.f;
      }
#pragma unroll
      for (int v = 0; v < V; ++v) {
        const int i = k * V + v;
        float a = bs[i];
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) a = fmaf(wt[j][i], hist[j][i], a);
        a = fmaf(wt[TAPS - 1][i], cur[v], a);
#pragma unroll
        for (int j = 0; j < TAPS - 2; ++j) hist[j][i] = hist[j + 1][i];
        if (TAPS > 1) hist[TAPS - 2 >= 0 ? TAPS - 2 : 0][i] = cur[v];
        a = silu(a);
        if (sizeof(TA) == 2) a = __bfloat162float(__float2bfloat16_rn(a));  // the norm is that of the stored activations
        y[i] = a;
        if (c + v < width) ss = fmaf(a, a, ss);
      }
      if (c + V <= width) stv<V>(out, (row0 + r) * ldo + cc + c, y + k * V);
      else {
#pragma unroll
        for (int v = 0; v < V; ++v)
          if (c + v < width) st(out, (row0 + r) * ldo + cc + c + v, y[k * V + v]);
      }
    }
    if (sec.unit[s]) {
      ss = wsum(ss);
      if (lane == 0) inv[(row0 + r) * ldi + unit_base + g] = sec.scale[s] / sqrtf(ss + 1e-6f);
    }
  }
  if (r0 == 0 && K > 0) {  // owner of the slot: it becomes the inputs of the entry's last K rows
#pragma unroll
    for (int k = 0; k < NK; ++k)
#pragma unroll
      for (int v = 0; v < V; ++v) {
        const int c = k * 32 * V + lane * V + v;
        if (c >= width) continue;
        for (int j = 0; j < K; ++j) {  // ascending: slot row n + j is read before it is overwritten
          const int row = n - K + j;
          float h = 0.f;
          if (row >= 0) h = ld(x, (row0 + row) * ldx + xc + c);
          else if (entry_ctx[e] > 0) h = slot[(long long)(n + j) * C + c];
          slot[(long long)j * C + c] = h;
        }
      }
  }
}

// The same for groups of V * 2^k <= 32 V channels and aligned rows (bf16; V = 4 or 8 channels per lane): a warp covers 32 V adjacent channels of a
// row (several groups), the next AHEAD rows are in flight while the current ones are computed, and AHEAD rows pass without a branch.
template <int V>
struct Packed;
template <>
struct Packed<4> { using T = uint2; };
template <>
struct Packed<8> { using T = uint4; };
__device__ __forceinline__ void unpack(uint2 u, float* v) {
  v[0] = __uint_as_float(u.x << 16); v[1] = __uint_as_float(u.x & 0xffff0000u);
  v[2] = __uint_as_float(u.y << 16); v[3] = __uint_as_float(u.y & 0xffff0000u);
}
__device__ __forceinline__ void unpack(uint4 u, float* v) {
  unpack(make_uint2(u.x, u.y), v);
  unpack(make_uint2(u.z, u.w), v + 4);
}
__device__ __forceinline__ void pack(const float* v, uint2& u) { u = make_uint2(pg::pack_bf16(v[0], v[1]), pg::pack_bf16(v[2], v[3])); }
__device__ __forceinline__ void pack(const float* v, uint4& u) {
  u = make_uint4(pg::pack_bf16(v[0], v[1]), pg::pack_bf16(v[2], v[3]), pg::pack_bf16(v[4], v[5]), pg::pack_bf16(v[6], v[7]));
}

template <int TAPS, int V>
__global__ void __launch_bounds__(128) short_conv_vec_kernel(const bf16* __restrict__ x, long long ldx, const float* __restrict__ w,
                                                             const float* __restrict__ bias, float* __restrict__ state, bf16* __restrict__ out,
                                                             long long ldo, float* __restrict__ inv, int ldi, PgConvSections sec, int taps, int C,
                                                             const int* __restrict__ entry_row0, const int* __restrict__ entry_n,
                                                             const int* __restrict__ entry_ctx, const int* __restrict__ entry_slot, int chunk) {
  constexpr int AHEAD = 4, WC = 32 * V;
  using P = typename Packed<V>::T;
  const int e = blockIdx.z, lane = threadIdx.x & 31;
  const int n = entry_n[e], r0 = blockIdx.y * chunk;
  if (r0 >= n) return;
  int g = blockIdx.x * 4 + (threadIdx.x >> 5), s = 0, unit_base = 0;
  while (s < sec.count && g >= (sec.total[s] + WC - 1) / WC) {
    g -= (sec.total[s] + WC - 1) / WC;
    if (sec.unit[s]) unit_base += sec.groups[s];
    ++s;
  }
  if (s >= sec.count) return;
  const int c = g * WC + lane * V;    // channel inside the section
  const bool ok = c < sec.total[s];   // totals are multiples of V
  const int lanes = sec.size[s] / V;  // lanes of one group
  const long long row0 = entry_row0[e];
  const bf16* xp = x + row0 * ldx + sec.xcol[s] + (ok ? c : 0);
  bf16* op = out + row0 * ldo + sec.ccol[s] + (ok ? c : 0);
  const int cc = sec.ccol[s] + (ok ? c : 0), K = taps - 1;
  float* slot = state + (long long)entry_slot[e] * K * C + cc;
  float wt[TAPS][V], bs[V], hist[TAPS - 1][V];
  auto ldf = [](const float* p, float* v) {
#pragma unroll
    for (int i = 0; i < V; i += 4) ldv<4>(p, i, v + i);
  };
  auto zero = [](float* v) {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = 0.f;
  };
  auto row_at = [&](int r) { return *reinterpret_cast<const P*>(xp + (long long)r * ldx); };
  if (bias != nullptr) ldf(bias + cc, bs); else zero(bs);
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    const int tj = j - (TAPS - taps);
    if (tj >= 0) ldf(w + (long long)tj * C + cc, wt[j]); else zero(wt[j]);
  }
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int row = r0 - (TAPS - 1) + j;
    if (row >= 0) unpack(row_at(row), hist[j]);
    else if (entry_ctx[e] > 0 && K + row >= 0) ldf(slot + (long long)(K + row) * C, hist[j]);
    else zero(hist[j]);
  }
  const int r1 = min(n, r0 + chunk);
  const bool unit = sec.unit[s] != 0;
  const float unit_scale = sec.scale[s];
  float* ip = (unit && ok && (lane & (lanes - 1)) == 0) ? inv + row0 * ldi + unit_base + c / sec.size[s] : nullptr;
  P nxt[AHEAD];
#pragma unroll
  for (int i = 0; i < AHEAD; ++i) nxt[i] = row_at(min(r0 + i, r1 - 1));
  for (int rb = r0; rb < r1; rb += AHEAD) {
    float ss[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int r = rb + i;  // rows past the run are computed from a repeated row and not stored
      float cur[V], y[V];
      unpack(nxt[i], cur);
      nxt[i] = row_at(min(r + AHEAD, r1 - 1));
#pragma unroll
      for (int v = 0; v < V; ++v) {
        float a = fmaf(wt[TAPS - 1][v], cur[v], bs[v]);
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) a = fmaf(wt[j][v], hist[j][v], a);
#pragma unroll
        for (int j = 0; j < TAPS - 2; ++j) hist[j][v] = hist[j + 1][v];
        hist[TAPS - 2][v] = cur[v];
        y[v] = __fdividef(a, 1.0f + __expf(-a));  // a bf16 activation: the hardware exponential is far below its rounding
      }
      P pk;
      pack(y, pk);
      if (ok && r < r1) *reinterpret_cast<P*>(op + (long long)r * ldo) = pk;
      unpack(pk, y);  // the norm is that of the stored activations
      ss[i] = 0.f;
#pragma unroll
      for (int v = 0; v < V; ++v) ss[i] = fmaf(y[v], y[v], ss[i]);
    }
    if (unit) {
      for (int o = lanes / 2; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
      if (ip != nullptr) {
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
          if (rb + i < r1) ip[(long long)(rb + i) * ldi] = unit_scale / sqrtf(ss[i] + 1e-6f);
      }
    }
  }
  if (r0 == 0 && K > 0 && ok) {  // owner of the slot: it becomes the inputs of the entry's last K rows
    for (int j = 0; j < K; ++j) {
      const int row = n - K + j;
      float h[V];
      if (row >= 0) unpack(row_at(row), h);
      else if (entry_ctx[e] > 0) ldf(slot + (long long)(n + j) * C, h);
      else zero(h);
#pragma unroll
      for (int i = 0; i < V; i += 4) stv<4>(slot, (long long)j * C + i, h + i);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------------
// Scans.  CTA = (block of 16 * VEC value columns, head, entry); thread = VEC value columns (ct) x every 16th key dimension (grp), its
// part of the state in registers.  Per token the key-side vectors go through shared memory (double-buffered) and the sums
// over the key dimension through a [16][16 * VEC] exchange area (double-buffered: two barriers per sum).
// ---------------------------------------------------------------------------------------------------------------------
template <typename TA, int VEC, int RP>
__global__ void __launch_bounds__(256) delta_scan_kernel(PgDeltaArgs a, int n_min, int n_max) {
  constexpr int VB = 16 * VEC;
  const int e = blockIdx.z, h = blockIdx.y;
  const int n = a.entry_n[e];
  if (n < n_min || n > n_max) return;
  const int dim = a.dim, vdim = a.vdim, H = a.H;
  const int ct = threadIdx.x & 15, grp = threadIdx.x >> 4;
  const int v0 = blockIdx.x * VB + ct * VEC;
  const bool v_ok = v0 < vdim;  // VEC 4: vdim is a multiple of 4
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;               // [2][dim]
  float* ks = qs + 2 * dim;     // [2][dim]
  float* gs = ks + 2 * dim;     // [2][dim]
  float* red = gs + 2 * dim;    // [2][16][VB]
  float* red2 = red + 32 * VB;  // [2][16][VB]
  float S[RP][VEC];
  float* stp = a.state + (((long long)a.entry_slot[e] * H + h) * dim) * vdim;
  const bool fresh = a.entry_ctx[e] == 0;
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int d = grp + 16 * i;
    if (!fresh && d < dim && v_ok) ldv<VEC>(stp, (long long)d * vdim + v0, S[i]);
    else {
#pragma unroll
      for (int v = 0; v < VEC; ++v) S[i][v] = 0.f;
    }
  }
  const int hk = h / (H / a.G);
  const TA* q = static_cast<const TA*>(a.q);
  const TA* k = static_cast<const TA*>(a.k);
  const TA* vv = static_cast<const TA*>(a.v);
  const TA* bl = static_cast<const TA*>(a.beta);
  const float rate = expf(a.A_log[h]);
  for (int t = 0; t < n; ++t) {
    const long long row = (long long)a.entry_row0[e] + t;
    const int bf = t & 1;
    const float iq = a.inv[row * a.ldi + hk], ik = a.inv[row * a.ldi + a.G + hk];
    for (int d = threadIdx.x; d < dim; d += 256) {
      qs[bf * dim + d] = ld(q, row * a.ldq + (long long)hk * dim + d) * iq;
      ks[bf * dim + d] = ld(k, row * a.ldk + (long long)hk * dim + d) * ik;
      gs[bf * dim + d] = expf(-rate * softplus(a.decay[row * a.lda + (long long)h * dim + d] + a.dt_bias[(long long)h * dim + d]));
    }
    float val[VEC];
    if (v_ok) ldv<VEC>(vv, row * a.ldv + (long long)h * vdim + v0, val);
    else {
#pragma unroll
      for (int v = 0; v < VEC; ++v) val[v] = 0.f;
    }
    const float beta = sigmoid(ld(bl, row * a.ldb + h));
    __syncthreads();
    float part[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) part[v] = 0.f;
#pragma unroll
    for (int i = 0; i < RP; ++i) {
      const int d = grp + 16 * i;
      if (d < dim) {
        const float g = gs[bf * dim + d], kd = ks[bf * dim + d];
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          S[i][v] *= g;
          part[v] = fmaf(S[i][v], kd, part[v]);
        }
      }
    }
    stv<VEC>(red, (bf * 16 + grp) * VB + ct * VEC, part);
    __syncthreads();
    float u[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) u[v] = 0.f;
#pragma unroll
    for (int p = 0; p < 16; ++p) {
      float r[VEC];
      ldv<VEC>(red, (bf * 16 + p) * VB + ct * VEC, r);
#pragma unroll
      for (int v = 0; v < VEC; ++v) u[v] += r[v];
    }
#pragma unroll
    for (int v = 0; v < VEC; ++v) {
      u[v] = beta * (val[v] - u[v]);
      part[v] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < RP; ++i) {
      const int d = grp + 16 * i;
      if (d < dim) {
        const float qd = qs[bf * dim + d], kd = ks[bf * dim + d];
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          S[i][v] = fmaf(kd, u[v], S[i][v]);
          part[v] = fmaf(S[i][v], qd, part[v]);
        }
      }
    }
    stv<VEC>(red2, (bf * 16 + grp) * VB + ct * VEC, part);
    __syncthreads();
    for (int c = threadIdx.x; c < VB; c += 256) {
      float o = 0.f;
#pragma unroll
      for (int p = 0; p < 16; ++p) o += red2[(bf * 16 + p) * VB + c];
      const int col = blockIdx.x * VB + c;
      if (col < vdim) a.out[row * ((long long)H * vdim) + (long long)h * vdim + col] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int d = grp + 16 * i;
    if (d < dim && v_ok) stv<VEC>(stp, (long long)d * vdim + v0, S[i]);
  }
}

// KIND 0: state space.  KIND 1: matrix memory; the normaliser n [dim] and the running maximum m of a head are kept once per block
// of value columns (norm_state [slots, blocks, H, dim + 1], m last), so that the CTAs of one head share no slot.
template <typename TA, int VEC, int RP, int KIND>
__global__ void __launch_bounds__(256) gated_scan_kernel(PgGatedArgs a, int n_min, int n_max) {
  constexpr int VB = 16 * VEC;
  const int e = blockIdx.z, h = blockIdx.y;
  const int n = a.entry_n[e];
  if (n < n_min || n > n_max) return;
  const int dim = a.dim, vdim = a.vdim, H = a.H;
  const int ct = threadIdx.x & 15, grp = threadIdx.x >> 4;
  const int v0 = blockIdx.x * VB + ct * VEC;
  const bool v_ok = v0 < vdim;
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;              // [2][dim]
  float* ks = qs + 2 * dim;    // [2][dim]
  float* red = ks + 2 * dim;   // [2][16][VB]
  float* redn = red + 32 * VB; // [2][16]
  float S[RP][VEC], nn[RP], m = 0.f;
  float* stp = a.state + (((long long)a.entry_slot[e] * H + h) * dim) * vdim;
  float* nst = KIND == 1 ? a.norm_state + (((long long)a.entry_slot[e] * gridDim.x + blockIdx.x) * H + h) * (dim + 1) : nullptr;
  const bool fresh = a.entry_ctx[e] == 0;
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int d = grp + 16 * i;
    if (!fresh && d < dim && v_ok) ldv<VEC>(stp, (long long)d * vdim + v0, S[i]);
    else {
#pragma unroll
      for (int v = 0; v < VEC; ++v) S[i][v] = 0.f;
    }
    nn[i] = (KIND == 1 && !fresh && d < dim) ? nst[d] : 0.f;
  }
  if (KIND == 1 && !fresh) m = nst[dim];
  const int hk = h / (H / a.G);
  const TA* q = static_cast<const TA*>(a.q);
  const TA* k = static_cast<const TA*>(a.k);
  const TA* vv = static_cast<const TA*>(a.v);
  const TA* g1 = static_cast<const TA*>(a.gate1);
  const TA* g2 = static_cast<const TA*>(a.gate2);
  const float c1 = a.p1[h], c2 = a.p2[h];
  const float rate = KIND == 0 ? expf(c2) : 0.f, skip = KIND == 0 ? a.p3[h] : 0.f;
  __syncthreads();  // m of the slot has been read by every thread before any is written (same CTA)
  for (int t = 0; t < n; ++t) {
    const long long row = (long long)a.entry_row0[e] + t;
    const int bf = t & 1;
    for (int d = threadIdx.x; d < dim; d += 256) {
      qs[bf * dim + d] = ld(q, row * a.ldq + (long long)hk * dim + d) * a.qscale;
      ks[bf * dim + d] = ld(k, row * a.ldk + (long long)hk * dim + d);
    }
    float val[VEC];
    if (v_ok) ldv<VEC>(vv, row * a.ldv + (long long)h * vdim + v0, val);
    else {
#pragma unroll
      for (int v = 0; v < VEC; ++v) val[v] = 0.f;
    }
    float keep, put;
    if (KIND == 0) {
      const float dt = softplus(ld(g1, row * a.ldg + h) + c1);
      keep = expf(-rate * dt);
      put = dt;
    } else {
      const float li = a.cap * tanhf((ld(g1, row * a.ldg + h) + c1) / a.cap);
      const float lf = -softplus(-a.cap * tanhf((ld(g2, row * a.ldg + h) + c2) / a.cap));
      const float mn = fmaxf(lf + m, li);
      keep = expf(lf + m - mn);
      put = expf(li - mn);
      m = mn;
    }
    float wv[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) wv[v] = put * val[v];
    __syncthreads();
    float part[VEC], pn = 0.f;
#pragma unroll
    for (int v = 0; v < VEC; ++v) part[v] = 0.f;
#pragma unroll
    for (int i = 0; i < RP; ++i) {
      const int d = grp + 16 * i;
      if (d < dim) {
        const float qd = qs[bf * dim + d], kd = ks[bf * dim + d];
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
          S[i][v] = fmaf(kd, wv[v], keep * S[i][v]);
          part[v] = fmaf(S[i][v], qd, part[v]);
        }
        if (KIND == 1) {
          nn[i] = fmaf(put, kd, keep * nn[i]);
          pn = fmaf(nn[i], qd, pn);
        }
      }
    }
    stv<VEC>(red, (bf * 16 + grp) * VB + ct * VEC, part);
    if (KIND == 1 && ct == 0) redn[bf * 16 + grp] = pn;
    __syncthreads();
    for (int c = threadIdx.x; c < VB; c += 256) {
      float o = 0.f;
#pragma unroll
      for (int p = 0; p < 16; ++p) o += red[(bf * 16 + p) * VB + c];
      const int col = blockIdx.x * VB + c;
      if (col < vdim) {
        if (KIND == 0) o = fmaf(skip, ld(vv, row * a.ldv + (long long)h * vdim + col), o);
        else {
          float nq = 0.f;
#pragma unroll
          for (int p = 0; p < 16; ++p) nq += redn[bf * 16 + p];
          o /= fmaxf(fabsf(nq), expf(-m)) + 1e-6f;
        }
        a.out[row * ((long long)H * vdim) + (long long)h * vdim + col] = o;
      }
    }
  }
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int d = grp + 16 * i;
    if (d < dim && v_ok) stv<VEC>(stp, (long long)d * vdim + v0, S[i]);
    if (KIND == 1 && d < dim && ct == 0) nst[d] = nn[i];
  }
  if (KIND == 1 && threadIdx.x == 0) nst[dim] = m;
}

// ---------------------------------------------------------------------------------------------------------------------
// out[t, :] = scale * gate(group-RMS-norm(o[t, :]) * w).  gate_mode 1: the normalised row times sigmoid(gate); 2: the row times
// silu(gate) BEFORE the norm.  w has one weight per column, or (w_n == group size) one per column of a group, shared by the groups.
// One CTA per row; with at least 8 groups a warp takes whole groups, else 8 / groups warps share one (when that divides).
// ---------------------------------------------------------------------------------------------------------------------
template <typename TA, int V>
__global__ void __launch_bounds__(256) group_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ w, int w_n,
                                                              const TA* __restrict__ gate, long long ldg, int gate_mode, TA* __restrict__ out,
                                                              long long ldo, int D, int groups, float eps, float scale) {
  __shared__ float red[8];
  const long long t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gs = D / groups;
  const int wpg = (groups < 8 && 8 % groups == 0) ? 8 / groups : 1;
  const int part = warp % wpg, stride = 32 * wpg * V;
  for (int g0 = warp / wpg; g0 < ((groups + 8 / wpg - 1) / (8 / wpg)) * (8 / wpg); g0 += 8 / wpg) {
    const bool g_ok = g0 < groups;
    const long long base = (long long)g0 * gs;
    float s = 0.f;
    if (g_ok)
      for (int d = (part * 32 + lane) * V; d < gs; d += stride) {
        float v[V], z[V];
        ldv<V>(o, t * D + base + d, v);
        if (gate_mode == 2) ldv<V>(gate, t * ldg + base + d, z);
#pragma unroll
        for (int i = 0; i < V; ++i) {
          if (gate_mode == 2) v[i] *= silu(z[i]);
          s = fmaf(v[i], v[i], s);
        }
      }
    s = wsum(s);
    if (wpg > 1) {
      __syncthreads();
      if (lane == 0) red[warp] = s;
      __syncthreads();
      s = 0.f;
      for (int p = 0; p < wpg; ++p) s += red[(warp / wpg) * wpg + p];
    }
    if (!g_ok) continue;
    const float iv = scale / sqrtf(s / (float)gs + eps);
    for (int d = (part * 32 + lane) * V; d < gs; d += stride) {
      float v[V], z[V], ww[V];
      ldv<V>(o, t * D + base + d, v);
      if (gate_mode != 0) ldv<V>(gate, t * ldg + base + d, z);
      if (w != nullptr) ldv<V>(w, w_n == gs ? d : base + d, ww);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        if (gate_mode == 2) v[i] *= silu(z[i]);
        v[i] *= w != nullptr ? iv * ww[i] : iv;
        if (gate_mode == 1) v[i] *= sigmoid(z[i]);
        if (gate_mode == 3) v[i] *= silu(z[i]);
      }
      stv<V>(out, t * ldo + base + d, v);
    }
  }
}

// Groups of 4 * NV * 2^k columns whose lanes fit a warp: lane <-> NV float4 of one group, several groups per warp, the row read once.
__device__ __forceinline__ float fast_sigmoid(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }

template <typename TA, int NV>
__global__ void __launch_bounds__(256) group_norm_gate_flat_kernel(const float* __restrict__ o, const float* __restrict__ w, int w_n,
                                                                   const TA* __restrict__ gate, long long ldg, int gate_mode, TA* __restrict__ out,
                                                                   long long ldo, int D, int gs, long long total_groups, float eps, float scale) {
  const int lanes = gs / (4 * NV), groups = D / gs;
  const long long id = (long long)blockIdx.x * (256 / lanes) + threadIdx.x / lanes;  // (row, group)
  const int l = threadIdx.x & (lanes - 1);
  const bool ok = id < total_groups;
  const long long t = ok ? id / groups : 0;
  const int col0 = (ok ? (int)(id % groups) : 0) * gs;
  float v[NV][4], z[NV][4], s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = col0 + (i * lanes + l) * 4;
    if (ok) {
      ldv<4>(o, t * D + d, v[i]);
      if (gate_mode != 0) ldv<4>(gate, t * ldg + d, z[i]);
    } else {
#pragma unroll
      for (int k = 0; k < 4; ++k) v[i][k] = z[i][k] = 0.f;
    }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      if (gate_mode != 0) {
        const float sg = sizeof(TA) == 2 ? fast_sigmoid(z[i][k]) : sigmoid(z[i][k]);
        if (gate_mode == 2) v[i][k] *= z[i][k] * sg;
        z[i][k] = gate_mode == 3 ? z[i][k] * sg : sg;
      }
      s = fmaf(v[i][k], v[i][k], s);
    }
  for (int x = lanes / 2; x > 0; x >>= 1) s += __shfl_xor_sync(0xffffffffu, s, x);
  if (!ok) return;
  const float iv = scale / sqrtf(s / (float)gs + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int in = (i * lanes + l) * 4;
    float ww[4];
    if (w != nullptr) ldv<4>(w, w_n == gs ? in : col0 + in, ww);
#pragma unroll
    for (int k = 0; k < 4; ++k) v[i][k] *= (w != nullptr ? iv * ww[k] : iv) * ((gate_mode & 1) ? z[i][k] : 1.0f);
    stv<4>(out, t * ldo + col0 + in, v[i]);
  }
}

inline bool al(const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

template <typename TA, int V, int NK, int TAPS>
int launch_conv(const void* x, long long ldx, const float* w, const float* bias, float* state, void* out, long long ldo, float* inv, int ldi,
                const PgConvSections& sec, int taps, int C, const int* row0, const int* n, const int* ctx, const int* slot, int entries, int max_n,
                cudaStream_t st) {
  int groups = 0;
  for (int s = 0; s < sec.count; ++s) groups += sec.groups[s];
  // long portions: runs of 32 rows, shortened while the launch would not fill the GPU twice over
  int chunk = 32;
  while (chunk > 8 && (long long)groups * entries * ((max_n + chunk - 1) / chunk) < 16LL * pg::num_sms()) chunk /= 2;
  const dim3 grid((groups + 3) / 4, (max_n + chunk - 1) / chunk, entries);
  short_conv_kernel<TA, V, NK, TAPS><<<grid, 128, 0, st>>>(static_cast<const TA*>(x), ldx, w, bias, state, static_cast<TA*>(out), ldo, inv, ldi, sec, taps, C,
                                                            row0, n, ctx, slot, chunk);
  PG_RET();
}

// V channels per lane (4 or 8; 0: only the general kernel fits): every group V * 2^k channels of at most 32 V, everything aligned
inline int conv_vec_width(const void* x, long long ldx, const float* w, const float* bias, const float* state, const void* out, long long ldo, int C,
                          const PgConvSections& sec) {
  if (!al(x, 16) || !al(out, 16) || !al(w, 16) || !al(bias, 16) || !al(state, 16) || ldx % 8 || ldo % 8 || C % 8) return 0;
  for (int v = 4; v <= 8; v += 4) {
    bool ok = true;
    for (int s = 0; s < sec.count; ++s) {
      const int l = sec.size[s] / v;
      ok = ok && sec.size[s] % v == 0 && l > 0 && l <= 32 && (l & (l - 1)) == 0 && sec.total[s] % v == 0 && sec.xcol[s] % 8 == 0 && sec.ccol[s] % 8 == 0;
    }
    if (ok) return v;
  }
  return 0;
}

template <int TAPS, int V>
int launch_conv_vec(const void* x, long long ldx, const float* w, const float* bias, float* state, void* out, long long ldo, float* inv, int ldi,
                    const PgConvSections& sec, int taps, int C, const int* row0, const int* n, const int* ctx, const int* slot, int entries, int max_n,
                    cudaStream_t st) {
  int warps = 0;
  for (int s = 0; s < sec.count; ++s) warps += (sec.total[s] + 32 * V - 1) / (32 * V);
  int chunk = 64;
  while (chunk > 8 && (long long)warps * entries * ((max_n + chunk - 1) / chunk) < 48LL * pg::num_sms()) chunk /= 2;
  const dim3 grid((warps + 3) / 4, (max_n + chunk - 1) / chunk, entries);
  short_conv_vec_kernel<TAPS, V><<<grid, 128, 0, st>>>(static_cast<const bf16*>(x), ldx, w, bias, state, static_cast<bf16*>(out), ldo, inv, ldi, sec, taps, C, row0,
                                                        n, ctx, slot, chunk);
  PG_RET();
}

template <typename TA, int TAPS>
int conv_shape(const void* x, long long ldx, const float* w, const float* bias, float* state, void* out, long long ldo, float* inv, int ldi,
               const PgConvSections& sec, int taps, int C, const int* row0, const int* n, const int* ctx, const int* slot, int entries, int max_n,
               cudaStream_t st) {
  int mx = 0;
  bool even = ldx % 2 == 0 && ldo % 2 == 0 && al(x, 8) && al(out, 8);
  for (int s = 0; s < sec.count; ++s) {
    mx = sec.size[s] > mx ? sec.size[s] : mx;
    even = even && sec.size[s] % 2 == 0 && sec.xcol[s] % 2 == 0 && sec.ccol[s] % 2 == 0;
  }
#define PG_CONV(V, NK) return launch_conv<TA, V, NK, TAPS>(x, ldx, w, bias, state, out, ldo, inv, ldi, sec, taps, C, row0, n, ctx, slot, entries, max_n, st)
  if (even) {
    if (mx <= 64) PG_CONV(2, 1);
    if (mx <= 128) PG_CONV(2, 2);
    if (mx <= 256) PG_CONV(2, 4);
    PG_CONV(2, 8);
  }
  if (mx <= 64) PG_CONV(1, 2);
  PG_CONV(1, 16);
#undef PG_CONV
}

}  // namespace

extern "C" int pg_short_conv(const void* x, long long ldx, const float* w, const float* bias, float* state, void* out, long long ldo, float* inv,
                             int ldi, const PgConvSections* sec, int taps, int C, const int* entry_row0, const int* entry_n, const int* entry_ctx,
                             const int* entry_slot, int entries, int max_n, int act_f32, void* stream) {
  if (sec == nullptr || sec->count <= 0 || sec->count > 3 || taps < 1 || taps > 8 || C <= 0 || entries <= 0 || entries > 65535 || max_n <= 0) return PG_ERR_ARG;
  if (taps > 1 && state == nullptr) return PG_ERR_ARG;
  for (int s = 0; s < sec->count; ++s) {
    if (sec->groups[s] <= 0 || sec->size[s] <= 0 || sec->size[s] > 512 || (sec->unit[s] && inv == nullptr)) return PG_ERR_ARG;
    if (sec->total[s] > sec->groups[s] * sec->size[s] || sec->total[s] <= (sec->groups[s] - 1) * sec->size[s]) return PG_ERR_ARG;
  }
  if ((max_n + 7) / 8 > 65535) return PG_ERR_ARG;
  cudaStream_t s = PG_ST(stream);
#define PG_CV(TA, TAPS) return conv_shape<TA, TAPS>(x, ldx, w, bias, state, out, ldo, inv, ldi, *sec, taps, C, entry_row0, entry_n, entry_ctx, entry_slot, entries, max_n, s)
  if (act_f32) {
    if (taps <= 4) PG_CV(float, 4);
    PG_CV(float, 8);
  }
  const int vw = conv_vec_width(x, ldx, w, bias, state, out, ldo, C, *sec);
#define PG_CVV(TAPS, V) return launch_conv_vec<TAPS, V>(x, ldx, w, bias, state, out, ldo, inv, ldi, *sec, taps, C, entry_row0, entry_n, entry_ctx, entry_slot, entries, max_n, s)
  if (vw == 4 && taps <= 4) PG_CVV(4, 4);
  if (vw == 4) PG_CVV(8, 4);
  if (vw == 8 && taps <= 4) PG_CVV(4, 8);
  if (vw == 8) PG_CVV(8, 8);
#undef PG_CVV
  if (taps <= 4) PG_CV(bf16, 4);
  PG_CV(bf16, 8);
#undef PG_CV
}

namespace {

template <typename TA, int VEC, int RP>
int launch_delta_scan(const PgDeltaArgs& a, int n_min, int n_max, cudaStream_t st) {
  constexpr int VB = 16 * VEC;
  const size_t smem = ((size_t)6 * a.dim + 64 * VB) * sizeof(float);
  delta_scan_kernel<TA, VEC, RP><<<dim3((a.vdim + VB - 1) / VB, a.H, a.entries), 256, smem, st>>>(a, n_min, n_max);
  PG_RET();
}

template <typename TA, int VEC, int RP, int KIND>
int launch_gated_scan(const PgGatedArgs& a, int n_min, int n_max, cudaStream_t st) {
  constexpr int VB = 16 * VEC;
  const size_t smem = ((size_t)4 * a.dim + 32 * VB + 32) * sizeof(float);
  gated_scan_kernel<TA, VEC, RP, KIND><<<dim3((a.vdim + VB - 1) / VB, a.H, a.entries), 256, smem, st>>>(a, n_min, n_max);
  PG_RET();
}

template <typename TA, int VEC>
int delta_rows(const PgDeltaArgs& a, int n_min, int n_max, cudaStream_t st) {
  if (a.dim <= 64) return launch_delta_scan<TA, VEC, 4>(a, n_min, n_max, st);
  if (a.dim <= 128) return launch_delta_scan<TA, VEC, 8>(a, n_min, n_max, st);
  if (a.dim <= 256) return launch_delta_scan<TA, VEC, 16>(a, n_min, n_max, st);
  return launch_delta_scan<TA, VEC, 32>(a, n_min, n_max, st);
}

template <typename TA, int VEC, int KIND>
int gated_rows(const PgGatedArgs& a, int n_min, int n_max, cudaStream_t st) {
  if (a.dim <= 64) return launch_gated_scan<TA, VEC, 4, KIND>(a, n_min, n_max, st);
  if (a.dim <= 128) return launch_gated_scan<TA, VEC, 8, KIND>(a, n_min, n_max, st);
  if (a.dim <= 256) return launch_gated_scan<TA, VEC, 16, KIND>(a, n_min, n_max, st);
  return launch_gated_scan<TA, VEC, 32, KIND>(a, n_min, n_max, st);
}

}  // namespace

// Value columns per CTA of the recurrent mixers: also the granularity of the matrix memory's normaliser slots.
extern "C" int pg_recurrence_block(int vdim) { return vdim % 4 == 0 ? 64 : 16; }

extern "C" int pg_delta_scan(const PgDeltaArgs* a, int n_min, int n_max, int act_f32, void* stream) {
  if (a == nullptr || a->entries <= 0 || a->entries > 65535 || a->H <= 0 || a->H > 65535 || a->G <= 0 || a->H % a->G || a->dim <= 0 || a->dim > 512 || a->vdim <= 0)
    return PG_ERR_ARG;
  const bool v4 = a->vdim % 4 == 0 && al(a->state, 16) && al(a->v, act_f32 ? 16 : 8) && a->ldv % 4 == 0;
  if (a->vdim % 4 == 0 && !v4) return PG_ERR_ARG;
  cudaStream_t st = PG_ST(stream);
  if (act_f32) return v4 ? delta_rows<float, 4>(*a, n_min, n_max, st) : delta_rows<float, 1>(*a, n_min, n_max, st);
  return v4 ? delta_rows<bf16, 4>(*a, n_min, n_max, st) : delta_rows<bf16, 1>(*a, n_min, n_max, st);
}

extern "C" int pg_gated_scan(const PgGatedArgs* a, int kind, int n_min, int n_max, int act_f32, void* stream) {
  if (a == nullptr || a->entries <= 0 || a->entries > 65535 || a->H <= 0 || a->H > 65535 || a->G <= 0 || a->H % a->G || a->dim <= 0 || a->dim > 512 || a->vdim <= 0 ||
      (kind != 0 && kind != 1) || (kind == 1 && (a->norm_state == nullptr || a->gate2 == nullptr || !(a->cap > 0.f))) || (kind == 0 && a->p3 == nullptr))
    return PG_ERR_ARG;
  const bool v4 = a->vdim % 4 == 0 && al(a->state, 16) && al(a->v, act_f32 ? 16 : 8) && a->ldv % 4 == 0;
  if (a->vdim % 4 == 0 && !v4) return PG_ERR_ARG;
  cudaStream_t st = PG_ST(stream);
#define PG_GS(TA, VEC) return kind == 0 ? gated_rows<TA, VEC, 0>(*a, n_min, n_max, st) : gated_rows<TA, VEC, 1>(*a, n_min, n_max, st)
  if (act_f32) {
    if (v4) PG_GS(float, 4);
    PG_GS(float, 1);
  }
  if (v4) PG_GS(bf16, 4);
  PG_GS(bf16, 1);
#undef PG_GS
}

extern "C" int pg_group_norm_gate(const float* o, const float* w, int w_n, const void* gate, long long ldg, int gate_mode, void* out, long long ldo,
                                  int rows, int D, int groups, float eps, float scale, int act_f32, void* stream) {
  if (rows <= 0 || D <= 0 || groups <= 0 || D % groups || (w != nullptr && w_n != D && w_n != D / groups) || gate_mode < 0 || gate_mode > 3 || (gate_mode && gate == nullptr))
    return PG_ERR_ARG;
  const int gs = D / groups, ab = act_f32 ? 4 : 2;
  auto fits = [&](int v) {
    return gs % v == 0 && ldg % v == 0 && ldo % v == 0 && al(o, 4 * v) && al(w, 4 * v) && al(gate, ab * v) && al(out, ab * v);
  };
  cudaStream_t st = PG_ST(stream);
  if (fits(4)) {
    const long long total = (long long)rows * groups;
    for (int nv = 1; nv <= 8; nv *= 2) {
      const int lanes = gs / (4 * nv);
      if (lanes * 4 * nv != gs || lanes > 32 || (lanes & (lanes - 1))) continue;
      const unsigned blocks = (unsigned)((total + 256 / lanes - 1) / (256 / lanes));
#define PG_GF(TA, NV) group_norm_gate_flat_kernel<TA, NV><<<blocks, 256, 0, st>>>(o, w, w_n, static_cast<const TA*>(gate), ldg, gate_mode, static_cast<TA*>(out), ldo, D, gs, total, eps, scale)
      if (act_f32) { if (nv == 1) PG_GF(float, 1); else if (nv == 2) PG_GF(float, 2); else if (nv == 4) PG_GF(float, 4); else PG_GF(float, 8); }
      else { if (nv == 1) PG_GF(bf16, 1); else if (nv == 2) PG_GF(bf16, 2); else if (nv == 4) PG_GF(bf16, 4); else PG_GF(bf16, 8); }
#undef PG_GF
      PG_RET();
    }
  }
#define PG_GN(TA, V) group_norm_gate_kernel<TA, V><<<rows, 256, 0, st>>>(o, w, w_n, static_cast<const TA*>(gate), ldg, gate_mode, static_cast<TA*>(out), ldo, D, groups, eps, scale)
  if (act_f32) {
    if (gs >= 128 && fits(4)) PG_GN(float, 4);
    else if (fits(2)) PG_GN(float, 2);
    else PG_GN(float, 1);
  } else {
    if (gs >= 128 && fits(4)) PG_GN(bf16, 4);
    else if (fits(2)) PG_GN(bf16, 2);
    else PG_GN(bf16, 1);
  }
#undef PG_GN
  PG_RET();
}
