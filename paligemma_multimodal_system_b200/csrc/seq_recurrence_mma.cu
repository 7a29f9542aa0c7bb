// Block forms of the recurrent mixers (seq_recurrence.cu) for prompt portions in bf16, on the tensor cores, with every quantity of the
// recurrence at fp32 precision.
//
// A CTA advances 64 value columns of one head of one entry through all its new tokens, a block of C tokens at a time.  The state is
// held TRANSPOSED, S^T [value column, key dimension], as the fp32 accumulators of m16n8k16 tiles (warp = 16 value columns): two
// adjacent 8-column accumulator tiles are, element for element, the A operand of a 16-deep product step, so S^T enters the products that
// read it straight from registers.  fp32 operands are cut into three bf16 terms (8 + 8 + 8 mantissa bits) and multiplied term by term: three
// products against a bf16-exact operand, six against another cut one (the dropped ones lie below 2^-24).
//
// Scalar decay (state space, matrix memory), block rows i, j with keys k, queries q, values v and the weights of PgGatedArgs:
//   o_i = carry_i S^T q_i + sum_{j <= i} P_ij v_j,  P_ij = exp(row_i - col_j) w_j (q_i . k_j);    S' = carry_C S + sum_j upd_j k_j v_j^T
// with row, col cumulative log decays (the running maximum of the matrix memory is a prefix maximum of i_j - F_j).
//
// Delta rule with per-channel decay, blocks of 16, L_t the cumulative log decay of the block (per channel), kg = k e^L, qg = q e^L,
// ke = k e^(L_end - L):
//   A_ij = sum_d k_i k_j e^(L_i - L_j) (j < i),  B_ij = sum_d q_i k_j e^(L_i - L_j) (j <= i),  W = (I + diag(beta) A)^-1 diag(beta)
//   U = W (V - kg S);   O = qg S + B U;   S' = diag(e^(L_end)) S + ke^T U
// A, B, W do not involve the state: pg_delta_blocks computes them for all blocks in parallel; only the second line is sequential.  Every
// exponent is a difference of the form (later - earlier) <= 0: strong decays underflow to zero and never overflow.
#include "common.cuh"
#include "paligemma_b200.h"

using bf16 = __nv_bfloat16;
using pg::cp_async16;
using pg::ldmatrix_x4;
using pg::ldmatrix_x4_trans;
using pg::mma_bf16_16816;
using pg::smem_u32;

#define PG_ST(s) reinterpret_cast<cudaStream_t>(s)

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float lo_f(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float hi_f(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }

// (p, q) = sum of three bf16 pairs, packed
__device__ __forceinline__ void cut3(float p, float q, uint32_t& a, uint32_t& b, uint32_t& c) {
  a = pg::pack_bf16(p, q);
  const float p1 = p - lo_f(a), q1 = q - hi_f(a);
  b = pg::pack_bf16(p1, q1);
  c = pg::pack_bf16(p1 - lo_f(b), q1 - hi_f(b));
}
// an accumulator pair of tiles -> the three A operands of a 16-deep step
__device__ __forceinline__ void cut_tiles(const float (&x)[4], const float (&y)[4], uint32_t (&a)[3][4]) {
  cut3(x[0], x[1], a[0][0], a[1][0], a[2][0]);
  cut3(x[2], x[3], a[0][1], a[1][1], a[2][1]);
  cut3(y[0], y[1], a[0][2], a[1][2], a[2][2]);
  cut3(y[2], y[3], a[0][3], a[1][3], a[2][3]);
}
// acc[i] += A B_i for a cut A and N cut B tiles (b0 / b1 = the halves of the B fragments, [tile][term]); consecutive products go to different
// accumulators, so that none waits for the one before it
template <int N>
__device__ __forceinline__ void mma6(float (&acc)[N][4], const uint32_t (&a)[3][4], const uint32_t (&b0)[N][3], const uint32_t (&b1)[N][3]) {
  constexpr int TA[6] = {0, 0, 1, 1, 0, 2}, TB[6] = {0, 1, 0, 1, 2, 0};
#pragma unroll
  for (int x = 0; x < 6; ++x)
#pragma unroll
    for (int i = 0; i < N; ++i) mma_bf16_16816(acc[i], a[TA[x]], b0[i][TB[x]], b1[i][TB[x]]);
}
// the same for two tiles with two partial sums each (four chains of three products)
__device__ __forceinline__ void mma6_pair(float (&acc)[2][4], const uint32_t (&a)[3][4], const uint4 (&f)[3]) {
  float lo[2][4] = {};
  const uint32_t b0[2][3] = {{f[0].x, f[1].x, f[2].x}, {f[0].z, f[1].z, f[2].z}}, b1[2][3] = {{f[0].y, f[1].y, f[2].y}, {f[0].w, f[1].w, f[2].w}};
  constexpr int HA[3] = {0, 1, 0}, HB[3] = {0, 0, 1}, LA[3] = {1, 0, 2}, LB[3] = {1, 2, 0};
#pragma unroll
  for (int x = 0; x < 3; ++x) {
#pragma unroll
    for (int i = 0; i < 2; ++i) mma_bf16_16816(acc[i], a[HA[x]], b0[i][HB[x]], b1[i][HB[x]]);
#pragma unroll
    for (int i = 0; i < 2; ++i) mma_bf16_16816(lo[i], a[LA[x]], b0[i][LB[x]], b1[i][LB[x]]);
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) acc[i][c] += lo[i][c];
}

// S^T fragments <-> the state slot [dim, vdim] (row pitch vdim): thread holds value columns v, v + 8 and key dimensions 8 nb + 2 tq, + 1
template <int DIM>
__device__ __forceinline__ void load_state(float (&S)[DIM / 8][4], const float* st, int dim, int vdim, int v, int tq, bool fresh) {
#pragma unroll
  for (int nb = 0; nb < DIM / 8; ++nb)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = nb * 8 + 2 * tq + (i & 1), c = v + (i >> 1) * 8;
      S[nb][i] = (!fresh && d < dim && c < vdim) ? st[(long long)d * vdim + c] : 0.f;
    }
}
template <int DIM>
__device__ __forceinline__ void store_state(const float (&S)[DIM / 8][4], float* st, int dim, int vdim, int v, int tq) {
#pragma unroll
  for (int nb = 0; nb < DIM / 8; ++nb)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = nb * 8 + 2 * tq + (i & 1), c = v + (i >> 1) * 8;
      if (d < dim && c < vdim) st[(long long)d * vdim + c] = S[nb][i];
    }
}

// ---------------------------------------------------------------------------------------------------------------------
// Scalar decay.  128 threads.  Per block: warp 0 turns the gates into the block's scalars (raw gates prefetched a block ahead), the
// q / k / v tiles arrive by cp.async a block ahead, warps w < C / 16 form 16 rows of P each, then every warp does its 16 value columns.
// ---------------------------------------------------------------------------------------------------------------------
template <int DIM, int C, int KIND>
__global__ void __launch_bounds__(128) gated_block_kernel(PgGatedArgs a, int n_min) {
  constexpr int LD = DIM + 8, LV = 64 + 8, LP = C + 8, TL = C / 32;  // TL: tokens per lane of warp 0
  const int e = blockIdx.z, h = blockIdx.y;
  const int n = a.entry_n[e];
  if (n < n_min) return;
  const int dim = a.dim, vdim = a.vdim, H = a.H;
  const long long row0 = a.entry_row0[e];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gq = lane >> 2, tq = lane & 3;
  extern __shared__ __align__(16) unsigned char smraw[];
  bf16* Qs = reinterpret_cast<bf16*>(smraw);  // [2][C][LD]
  bf16* Ks = Qs + 2 * C * LD;                 // [2][C][LD]
  bf16* Vs = Ks + 2 * C * LD;                 // [2][C][LV]
  bf16* Ps = Vs + 2 * C * LV;                 // [3][C][LP]
  float* sc = reinterpret_cast<float*>(Ps + 3 * C * LP);  // [2][5][C] row, col, w, carry, upd
  float* misc = sc + 2 * 5 * C;               // [2][2] carry of the whole block, m after the block's ...
  float* em = misc + 4;                       // [2][C] exp(-m) per token (matrix memory)
  float* den = em + 2 * C;                    // [C] 1 / denominator
  float* nv = den + C;                        // [DIM] normaliser
  const int hk = h / (H / a.G), v_base = blockIdx.x * 64, vcol = v_base + warp * 16 + gq;
  const bf16* q = static_cast<const bf16*>(a.q) + (long long)hk * dim;
  const bf16* k = static_cast<const bf16*>(a.k) + (long long)hk * dim;
  const bf16* vp = static_cast<const bf16*>(a.v) + (long long)h * vdim + v_base;
  const bf16* g1 = static_cast<const bf16*>(a.gate1) + h;
  const bf16* g2 = KIND == 1 ? static_cast<const bf16*>(a.gate2) + h : nullptr;
  float* stp = a.state + (((long long)a.entry_slot[e] * H + h) * dim) * vdim;
  float* nst = KIND == 1 ? a.norm_state + (((long long)a.entry_slot[e] * gridDim.x + blockIdx.x) * H + h) * (dim + 1) : nullptr;
  const bool fresh = a.entry_ctx[e] == 0;
  float S[DIM / 8][4];
  load_state<DIM>(S, stp, dim, vdim, vcol, tq, fresh);
  float m_run = 0.f;  // warp 0
  if (KIND == 1) {
    for (int d = threadIdx.x; d < DIM; d += 128) nv[d] = (!fresh && d < dim) ? nst[d] : 0.f;
    if (!fresh) m_run = nst[dim];
  }
  const float c1 = a.p1[h], c2 = a.p2[h], rate = KIND == 0 ? expf(c2) * LOG2E : 0.f, skip = KIND == 0 ? a.p3[h] : 0.f;
  float raw1[TL], raw2[TL];
  auto fetch_gates = [&](int t0) {
#pragma unroll
    for (int i = 0; i < TL; ++i) {
      const int t = t0 + lane * TL + i;
      raw1[i] = t < n ? __bfloat162float(g1[(row0 + t) * a.ldg]) : 0.f;
      raw2[i] = (KIND == 1 && t < n) ? __bfloat162float(g2[(row0 + t) * a.ldg]) : 0.f;
    }
  };
  auto fetch = [&](int t0, int buf) {
    for (int id = threadIdx.x; id < C * (DIM / 8); id += 128) {
      const int r = id / (DIM / 8), c = (id % (DIM / 8)) * 8;
      const bool ok = t0 + r < n && c < dim;
      const long long row = row0 + (ok ? t0 + r : 0);
      cp_async16(smem_u32(Qs + (buf * C + r) * LD + c), q + row * a.ldq + (ok ? c : 0), ok);
      cp_async16(smem_u32(Ks + (buf * C + r) * LD + c), k + row * a.ldk + (ok ? c : 0), ok);
    }
    for (int id = threadIdx.x; id < C * 8; id += 128) {
      const int r = id / 8, c = (id % 8) * 8;
      const bool ok = t0 + r < n && v_base + c < vdim;
      cp_async16(smem_u32(Vs + (buf * C + r) * LV + c), vp + (row0 + (ok ? t0 + r : 0)) * a.ldv + (ok ? c : 0), ok);
    }
    pg::cp_async_commit();
  };
  // lane's row / column inside a 16 x 16 block for ldmatrix: A operand (row-major), B operand (rows = n), and their transposed forms
  const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = ((lane >> 4) & 1) * 8;
  const int b_row = (lane & 7) + ((lane >> 4) & 1) * 8, b_col = ((lane >> 3) & 1) * 8;
  fetch(0, 0);
  if (warp == 0) fetch_gates(0);
  int cur = 0;
  for (int t0 = 0; t0 < n; t0 += C, cur ^= 1) {
    float* scb = sc + cur * 5 * C;
    if (warp == 0) {
      if (KIND == 0) {
        // cumulative log2 decay; tokens past the end: no decay, no write
        float dt[TL], L[TL], run = 0.f;
#pragma unroll
        for (int i = 0; i < TL; ++i) {
          const bool ok = t0 + lane * TL + i < n;
          dt[i] = ok ? softplus(raw1[i] + c1) : 0.f;
          run -= rate * dt[i];
          L[i] = run;
        }
        float pre = run;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float x = __shfl_up_sync(0xffffffffu, pre, o);
          if (lane >= o) pre += x;
        }
        const float tot = __shfl_sync(0xffffffffu, pre, 31);
        pre -= run;
#pragma unroll
        for (int i = 0; i < TL; ++i) {
          const int t = lane * TL + i;
          const float l = L[i] + pre;
          scb[t] = l;
          scb[C + t] = l;
          scb[2 * C + t] = dt[i];
          scb[3 * C + t] = exp2f(l);
          scb[4 * C + t] = exp2f(tot - l) * dt[i];
        }
        if (lane == 0) misc[cur * 2] = exp2f(tot);
      } else {
        // F: cumulative log forget gate; b = i - F; M: prefix maximum of b (and the old m); m_t = F_t + M_t   (natural logs)
        float F[TL], b[TL], run = 0.f;
#pragma unroll
        for (int i = 0; i < TL; ++i) {
          const bool ok = t0 + lane * TL + i < n;
          run += ok ? -softplus(-a.cap * tanhf((raw2[i] + c2) / a.cap)) : 0.f;
          F[i] = run;
          b[i] = ok ? a.cap * tanhf((raw1[i] + c1) / a.cap) : -1e30f;
        }
        float pre = run;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float x = __shfl_up_sync(0xffffffffu, pre, o);
          if (lane >= o) pre += x;
        }
        const float Ftot = __shfl_sync(0xffffffffu, pre, 31);
        pre -= run;
        float mx = -1e30f, M[TL];
#pragma unroll
        for (int i = 0; i < TL; ++i) {
          F[i] += pre;
          b[i] -= F[i];
          mx = fmaxf(mx, b[i]);
          M[i] = mx;
        }
        float pm = mx;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float x = __shfl_up_sync(0xffffffffu, pm, o);
          if (lane >= o) pm = fmaxf(pm, x);
        }
        float before = __shfl_up_sync(0xffffffffu, pm, 1);
        if (lane == 0) before = -1e30f;
        const float Mend = fmaxf(m_run, __shfl_sync(0xffffffffu, pm, 31));
#pragma unroll
        for (int i = 0; i < TL; ++i) {
          const int t = lane * TL + i;
          const float Mi = fmaxf(m_run, fmaxf(before, M[i]));
          scb[t] = -Mi * LOG2E;
          scb[C + t] = -b[i] * LOG2E;
          scb[2 * C + t] = a.qscale;
          scb[3 * C + t] = expf(m_run - Mi) * a.qscale;
          scb[4 * C + t] = expf(b[i] - Mend);
          em[cur * C + t] = expf(-(F[i] + Mi));
        }
        if (lane == 0) misc[cur * 2] = expf(m_run - Mend);
        m_run = Ftot + Mend;
      }
      fetch_gates(t0 + C);
    }
    pg::cp_async_wait<0>();
    __syncthreads();  // this block's tiles and scalars are there; every warp is done with the other buffers
    if (t0 + C < n) fetch(t0 + C, cur ^ 1);
    const bf16* Qb = Qs + cur * C * LD;
    const bf16* Kb = Ks + cur * C * LD;
    const bf16* Vb = Vs + cur * C * LV;
    // P: warp = rows 16 warp .. + 15
    if (warp < C / 16) {
      const int tl = warp * 16 + gq, th = tl + 8;
      const float row_l = scb[tl], row_h = scb[th];
      float sum_l = 0.f, sum_h = 0.f;
      uint32_t qa[DIM / 16][4];
#pragma unroll
      for (int kd = 0; kd < DIM / 16; ++kd) ldmatrix_x4(smem_u32(Qb + (warp * 16 + a_row) * LD + kd * 16 + a_col), qa[kd][0], qa[kd][1], qa[kd][2], qa[kd][3]);
      for (int jb = 0; jb <= warp; ++jb) {
        float s[2][4] = {};
#pragma unroll
        for (int kd = 0; kd < DIM / 16; ++kd) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(smem_u32(Kb + (jb * 16 + b_row) * LD + kd * 16 + b_col), b0, b1, b2, b3);
          mma_bf16_16816(s[0], qa[kd], b0, b1);
          mma_bf16_16816(s[1], qa[kd], b2, b3);
        }
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
          const int j = jb * 16 + nb * 8 + 2 * tq;
          const float2 col = *reinterpret_cast<const float2*>(scb + C + j), w = *reinterpret_cast<const float2*>(scb + 2 * C + j);
          float p[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int t = (i & 2) ? th : tl, key = j + (i & 1);
            const float x = exp2f(((i & 2) ? row_h : row_l) - ((i & 1) ? col.y : col.x)) * ((i & 1) ? w.y : w.x);
            p[i] = key <= t ? s[nb][i] * x : 0.f;
          }
          if (KIND == 1) { sum_l += p[0] + p[1]; sum_h += p[2] + p[3]; }
          uint32_t c[3][2];
          cut3(p[0], p[1], c[0][0], c[1][0], c[2][0]);
          cut3(p[2], p[3], c[0][1], c[1][1], c[2][1]);
#pragma unroll
          for (int x = 0; x < 3; ++x) {
            *reinterpret_cast<uint32_t*>(Ps + (x * C + tl) * LP + j) = c[x][0];
            *reinterpret_cast<uint32_t*>(Ps + (x * C + th) * LP + j) = c[x][1];
          }
        }
      }
      if (KIND == 1) {
        // n . q of the carried normaliser: the four lanes of a quad share a row pair
        float dl = 0.f, dh = 0.f;
#pragma unroll
        for (int kd = 0; kd < DIM / 16; ++kd) {
          const float2 n0 = *reinterpret_cast<const float2*>(nv + kd * 16 + 2 * tq), n1 = *reinterpret_cast<const float2*>(nv + kd * 16 + 8 + 2 * tq);
          dl += n0.x * lo_f(qa[kd][0]) + n0.y * hi_f(qa[kd][0]) + n1.x * lo_f(qa[kd][2]) + n1.y * hi_f(qa[kd][2]);
          dh += n0.x * lo_f(qa[kd][1]) + n0.y * hi_f(qa[kd][1]) + n1.x * lo_f(qa[kd][3]) + n1.y * hi_f(qa[kd][3]);
        }
        sum_l = fmaf(dl, scb[3 * C + tl], sum_l);
        sum_h = fmaf(dh, scb[3 * C + th], sum_h);
        sum_l += __shfl_xor_sync(0xffffffffu, sum_l, 1); sum_l += __shfl_xor_sync(0xffffffffu, sum_l, 2);
        sum_h += __shfl_xor_sync(0xffffffffu, sum_h, 1); sum_h += __shfl_xor_sync(0xffffffffu, sum_h, 2);
        if (tq == 0) {
          den[tl] = 1.0f / (fmaxf(fabsf(sum_l), em[cur * C + tl]) + 1e-6f);
          den[th] = 1.0f / (fmaxf(fabsf(sum_h), em[cur * C + th]) + 1e-6f);
        }
      }
    }
    __syncthreads();  // P (and the denominators) are complete
    // outputs O^T [16 value columns, C tokens]
    float o[C / 8][4];
#pragma unroll
    for (int i = 0; i < C / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
    for (int kd = 0; kd < DIM / 16; ++kd) {
      uint32_t sa[3][4];
      cut_tiles(S[2 * kd], S[2 * kd + 1], sa);
      uint32_t bq[C / 16][4];
#pragma unroll
      for (int tb = 0; tb < C / 16; ++tb) ldmatrix_x4(smem_u32(Qb + (tb * 16 + b_row) * LD + kd * 16 + b_col), bq[tb][0], bq[tb][1], bq[tb][2], bq[tb][3]);
#pragma unroll
      for (int x = 0; x < 3; ++x)  // consecutive products go to different accumulators
#pragma unroll
        for (int tb = 0; tb < C / 16; ++tb) {
          mma_bf16_16816(o[2 * tb], sa[x], bq[tb][0], bq[tb][1]);
          mma_bf16_16816(o[2 * tb + 1], sa[x], bq[tb][2], bq[tb][3]);
        }
    }
#pragma unroll
    for (int nb = 0; nb < C / 8; ++nb) {
      const float2 c = *reinterpret_cast<const float2*>(scb + 3 * C + nb * 8 + 2 * tq);
      o[nb][0] *= c.x; o[nb][1] *= c.y; o[nb][2] *= c.x; o[nb][3] *= c.y;
    }
#pragma unroll
    for (int kk = 0; kk < C / 16; ++kk) {
      uint32_t va[4];
      ldmatrix_x4_trans(smem_u32(Vb + (kk * 16 + b_row) * LV + warp * 16 + b_col), va[0], va[1], va[2], va[3]);
#pragma unroll
      for (int x = 0; x < 3; ++x)
#pragma unroll
        for (int tb = kk; tb < C / 16; ++tb) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(smem_u32(Ps + (x * C + tb * 16 + b_row) * LP + kk * 16 + b_col), b0, b1, b2, b3);
          mma_bf16_16816(o[2 * tb], va, b0, b1);
          mma_bf16_16816(o[2 * tb + 1], va, b2, b3);
        }
      if (KIND == 0) {  // the skip: token block kk of V^T has the accumulator's layout
        o[2 * kk][0] = fmaf(skip, lo_f(va[0]), o[2 * kk][0]); o[2 * kk][1] = fmaf(skip, hi_f(va[0]), o[2 * kk][1]);
        o[2 * kk][2] = fmaf(skip, lo_f(va[1]), o[2 * kk][2]); o[2 * kk][3] = fmaf(skip, hi_f(va[1]), o[2 * kk][3]);
        o[2 * kk + 1][0] = fmaf(skip, lo_f(va[2]), o[2 * kk + 1][0]); o[2 * kk + 1][1] = fmaf(skip, hi_f(va[2]), o[2 * kk + 1][1]);
        o[2 * kk + 1][2] = fmaf(skip, lo_f(va[3]), o[2 * kk + 1][2]); o[2 * kk + 1][3] = fmaf(skip, hi_f(va[3]), o[2 * kk + 1][3]);
      }
    }
#pragma unroll
    for (int nb = 0; nb < C / 8; ++nb)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = nb * 8 + 2 * tq + (i & 1), c = vcol + (i >> 1) * 8;
        float y = o[nb][i];
        if (KIND == 1) y *= den[t];
        if (t0 + t < n && c < vdim) a.out[(row0 + t0 + t) * ((long long)H * vdim) + (long long)h * vdim + c] = y;
      }
    // state
    const float carry = misc[cur * 2];
#pragma unroll
    for (int nb = 0; nb < DIM / 8; ++nb) { S[nb][0] *= carry; S[nb][1] *= carry; S[nb][2] *= carry; S[nb][3] *= carry; }
#pragma unroll
    for (int kk = 0; kk < C / 16; ++kk) {
      uint32_t va[4], wa[3][4];
      ldmatrix_x4_trans(smem_u32(Vb + (kk * 16 + b_row) * LV + warp * 16 + b_col), va[0], va[1], va[2], va[3]);
      const float2 u0 = *reinterpret_cast<const float2*>(scb + 4 * C + kk * 16 + 2 * tq), u1 = *reinterpret_cast<const float2*>(scb + 4 * C + kk * 16 + 8 + 2 * tq);
      cut3(lo_f(va[0]) * u0.x, hi_f(va[0]) * u0.y, wa[0][0], wa[1][0], wa[2][0]);
      cut3(lo_f(va[1]) * u0.x, hi_f(va[1]) * u0.y, wa[0][1], wa[1][1], wa[2][1]);
      cut3(lo_f(va[2]) * u1.x, hi_f(va[2]) * u1.y, wa[0][2], wa[1][2], wa[2][2]);
      cut3(lo_f(va[3]) * u1.x, hi_f(va[3]) * u1.y, wa[0][3], wa[1][3], wa[2][3]);
#pragma unroll
      for (int dp = 0; dp < DIM / 32; ++dp) {
        uint32_t bk[2][4];
#pragma unroll
        for (int hf = 0; hf < 2; ++hf)
          ldmatrix_x4_trans(smem_u32(Kb + (kk * 16 + a_row) * LD + (2 * dp + hf) * 16 + a_col), bk[hf][0], bk[hf][1], bk[hf][2], bk[hf][3]);
#pragma unroll
        for (int x = 0; x < 3; ++x)
#pragma unroll
          for (int hf = 0; hf < 2; ++hf) {
            mma_bf16_16816(S[4 * dp + 2 * hf], wa[x], bk[hf][0], bk[hf][1]);
            mma_bf16_16816(S[4 * dp + 2 * hf + 1], wa[x], bk[hf][2], bk[hf][3]);
          }
      }
    }
    if (KIND == 1) {  // every read of the old normaliser was before the barrier above; the next one follows the next barrier
      for (int d = threadIdx.x; d < DIM; d += 128) {
        float s = nv[d] * carry;
        for (int j = 0; j < C; ++j) s = fmaf(scb[4 * C + j], __bfloat162float(Kb[j * LD + d]), s);
        nv[d] = s;
      }
    }
  }
  store_state<DIM>(S, stp, dim, vdim, vcol, tq);
  if (KIND == 1) {
    for (int d = threadIdx.x; d < dim; d += 128) nst[d] = nv[d];  // the thread that wrote nv[d]
    if (threadIdx.x == 0) nst[dim] = m_run;
  }
}

// ---------------------------------------------------------------------------------------------------------------------
// Delta rule, the state-free part.  One CTA per (block of 16 tokens, head, entry): the cumulative log2 decays replace the raw ones in
// `decay`, and W and B leave as the B operands of 16-deep product steps, cut into three terms, in fragment order
// (scratch [block, head, {W, B}, term, lane] of uint4 = the halves of token columns 0-7, then 8-15).
// Inside a half block (8 tokens) the exponentials are taken per pair; between the halves they factor through the first half's end.
// ---------------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ long long block_index(const PgDeltaArgs& a, int e, int blk) { return a.entry_row0[e] / 16 + e + blk; }

template <int DIMP>
__global__ void __launch_bounds__(128) delta_blocks_kernel(PgDeltaArgs a, float* __restrict__ decay, uint4* __restrict__ scratch, int n_min) {
  constexpr int LD = DIMP + 4;
  const int e = blockIdx.z, h = blockIdx.y, blk = blockIdx.x;
  const int n = a.entry_n[e];
  if (n < n_min || blk * 16 >= n) return;
  const int dim = a.dim, cn = min(16, n - blk * 16);
  const long long row0 = (long long)a.entry_row0[e] + blk * 16;
  extern __shared__ __align__(16) float sm[];
  float* Lg = sm;              // [16][LD] log2 decay, cumulative inside the half block
  float* Kn = Lg + 16 * LD;    // [16][LD] k
  float* Qn = Kn + 16 * LD;    // [16][LD] q
  float* Kf = Qn + 16 * LD;    // [16][LD] k decayed to (first half) / from (second half) the first half's end
  float* Qf = Kf + 16 * LD;    // [8][LD]  q of the second half decayed from the first half's end
  float* Am = Qf + 8 * LD;     // [16][17]
  float* Bm = Am + 16 * 17;    // [16][17]
  float* Wm = Bm + 16 * 17;    // [16][17]
  float* bt = Wm + 16 * 17;    // [16]
  float* iv = bt + 16;         // [2][16] inverse norms of q, k
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int hk = h / (a.H / a.G);
  const bf16* q = static_cast<const bf16*>(a.q) + (long long)hk * dim;
  const bf16* k = static_cast<const bf16*>(a.k) + (long long)hk * dim;
  const float rate = -expf(a.A_log[h]) * LOG2E;
  for (int i = tid; i < 2 * 16 * 17; i += 128) Am[i] = 0.f;  // A and B
  if (tid < 16) {
    const bool ok = tid < cn;
    const float* ivr = a.inv + (row0 + tid) * a.ldi;
    bt[tid] = ok ? 1.0f / (1.0f + expf(-__bfloat162float(static_cast<const bf16*>(a.beta)[(row0 + tid) * a.ldb + h]))) : 0.f;
    iv[tid] = ok ? ivr[hk] : 0.f;
    iv[16 + tid] = ok ? ivr[a.G + hk] : 0.f;
  }
  constexpr int ITEMS = (2 * DIMP + 127) / 128;  // (half block, channel) pairs of a thread
  float lg[ITEMS][8];
  bf16 kr[ITEMS][8], qr[ITEMS][8];
  const bf16 zero = __float2bfloat16_rn(0.f);
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int item = tid + it * 128, half = item / DIMP, d = item % DIMP;
    const bool in = item < 2 * DIMP && d < dim;
    const int nt = in ? min(8, cn - half * 8) : 0;  // tokens of this half
    const long long r = row0 + half * 8;
    const bf16 *kp = k + r * a.ldk + d, *qp = q + r * a.ldq + d;
    const float* lp = decay + r * a.lda + (long long)h * dim + d;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const bool ok = i < nt;
      kr[it][i] = ok ? *kp : zero;
      qr[it][i] = ok ? *qp : zero;
      lg[it][i] = ok ? *lp : 0.f;
      kp += a.ldk;
      qp += a.ldq;
      lp += a.lda;
    }
  }
  __syncthreads();
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int item = tid + it * 128, half = item / DIMP, d = item % DIMP;
    if (item >= 2 * DIMP) break;
    const int nt = d < dim ? min(8, cn - half * 8) : 0;
    const float bias = d < dim ? a.dt_bias[(long long)h * dim + d] : 0.f;
    float run = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float z = lg[it][i] + bias;
      const float sp = fmaxf(z, 0.f) + log1pf(exp2f(-fabsf(z) * LOG2E));
      if (i < nt) run = fmaf(rate, sp, run);
      lg[it][i] = run;
    }
    const int o = half * 8 * LD + d;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float kv = __bfloat162float(kr[it][i]) * iv[16 + half * 8 + i], qv = __bfloat162float(qr[it][i]) * iv[half * 8 + i];
      Lg[o + i * LD] = lg[it][i];
      Kn[o + i * LD] = kv;
      Qn[o + i * LD] = qv;
      const float f = exp2f(half == 0 ? run - lg[it][i] : lg[it][i]);
      Kf[o + i * LD] = kv * f;
      if (half == 1) Qf[i * LD + d] = qv * f;
    }
  }
  __syncthreads();
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {  // cumulative over the block, for the sequential part
    const int item = tid + it * 128, half = item / DIMP, d = item % DIMP;
    if (item < 2 * DIMP && d < dim) {
      const int nt = min(8, cn - half * 8);
      const float base = half == 1 ? Lg[7 * LD + d] : 0.f;
      float* lp = decay + (row0 + half * 8) * a.lda + (long long)h * dim + d;
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i < nt) lp[i * a.lda] = lg[it][i] + base;
    }
  }
  if (warp < 2) {
    // strictly lower pairs of half block `warp`: lane -> (i, j), i > j
    if (lane < 28) {
      int i = 1, r = lane;
      while (r >= i) { r -= i; ++i; }
      const int t = warp * 8 + i, j = warp * 8 + r;
      float sa = 0.f, sb = 0.f;
      for (int d = 0; d < DIMP; d += 4) {
        const float4 lt = *reinterpret_cast<const float4*>(Lg + t * LD + d), lj = *reinterpret_cast<const float4*>(Lg + j * LD + d);
        const float4 kt = *reinterpret_cast<const float4*>(Kn + t * LD + d), kj = *reinterpret_cast<const float4*>(Kn + j * LD + d);
        const float4 qt = *reinterpret_cast<const float4*>(Qn + t * LD + d);
        const float e0 = exp2f(lt.x - lj.x) * kj.x, e1 = exp2f(lt.y - lj.y) * kj.y, e2 = exp2f(lt.z - lj.z) * kj.z, e3 = exp2f(lt.w - lj.w) * kj.w;
        sa = fmaf(kt.x, e0, fmaf(kt.y, e1, fmaf(kt.z, e2, fmaf(kt.w, e3, sa))));
        sb = fmaf(qt.x, e0, fmaf(qt.y, e1, fmaf(qt.z, e2, fmaf(qt.w, e3, sb))));
      }
      Am[t * 17 + j] = sa;
      Bm[t * 17 + j] = sb;
    }
  } else {
    const int id = (warp - 2) * 32 + lane, t = 8 + id / 8, j = id % 8;
    float sa = 0.f, sb = 0.f;
    for (int d = 0; d < DIMP; d += 4) {
      const float4 kj = *reinterpret_cast<const float4*>(Kf + j * LD + d), kt = *reinterpret_cast<const float4*>(Kf + t * LD + d);
      const float4 qt = *reinterpret_cast<const float4*>(Qf + (t - 8) * LD + d);
      sa = fmaf(kt.x, kj.x, fmaf(kt.y, kj.y, fmaf(kt.z, kj.z, fmaf(kt.w, kj.w, sa))));
      sb = fmaf(qt.x, kj.x, fmaf(qt.y, kj.y, fmaf(qt.z, kj.z, fmaf(qt.w, kj.w, sb))));
    }
    Am[t * 17 + j] = sa;
    Bm[t * 17 + j] = sb;
    if (lane < 8) {  // the diagonal of B has no decay
      const int td = (warp - 2) * 8 + lane;
      float s = 0.f;
      for (int d = 0; d < DIMP; d += 4) {
        const float4 kt = *reinterpret_cast<const float4*>(Kn + td * LD + d), qt = *reinterpret_cast<const float4*>(Qn + td * LD + d);
        s = fmaf(qt.x, kt.x, fmaf(qt.y, kt.y, fmaf(qt.z, kt.z, fmaf(qt.w, kt.w, s))));
      }
      Bm[td * 17 + td] = s;
    }
  }
  __syncthreads();
  uint4* dst = scratch + (block_index(a, e, blk) * a.H + h) * 6 * 32;
  const int gq = lane >> 2, tq = lane & 3;
  auto emit = [&](const float* Mx, uint4* to) {
    uint32_t f[3][4];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const float* p = Mx + (nb * 8 + gq) * 17 + hf * 8 + 2 * tq;
        cut3(p[0], p[1], f[0][nb * 2 + hf], f[1][nb * 2 + hf], f[2][nb * 2 + hf]);
      }
#pragma unroll
    for (int x = 0; x < 3; ++x) to[x * 32 + lane] = make_uint4(f[x][0], f[x][1], f[x][2], f[x][3]);
  };
  if (warp == 0) {
    // columns of (I + diag(beta) A)^-1 by forward substitution, one per lane
    if (lane < 16) {
      float x[16];
#pragma unroll
      for (int t = 0; t < 16; ++t) {
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < t; ++j) s = fmaf(Am[t * 17 + j], x[j], s);
        x[t] = (t == lane ? 1.0f : 0.f) - bt[t] * s;
        Wm[t * 17 + lane] = x[t] * bt[lane];
      }
    }
    __syncwarp();
    emit(Wm, dst);
  } else if (warp == 1) {
    emit(Bm, dst + 3 * 32);
  }
}

// ---------------------------------------------------------------------------------------------------------------------
// Delta rule, the sequential part.  128 threads, warp = 16 value columns.  The operand tiles kg, qg, ke of block b + 1 are formed (from
// q, k and cumulative decays fetched into registers a block earlier) while block b's tiles are multiplied; one barrier per block.
// ---------------------------------------------------------------------------------------------------------------------
template <int DIM>
__global__ void __launch_bounds__(128) delta_chain_kernel(PgDeltaArgs a, const uint4* __restrict__ scratch, int n_min) {
  constexpr int LD = DIM + 8, LV = 72, NI = (DIM + 63) / 64, TILE = 16 * LD;
  const int e = blockIdx.z, h = blockIdx.y;
  const int n = a.entry_n[e];
  if (n < n_min) return;
  const int dim = a.dim, vdim = a.vdim, H = a.H;
  const long long row0 = a.entry_row0[e];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, tq = lane & 3;
  extern __shared__ __align__(16) unsigned char smraw[];
  bf16* Tl = reinterpret_cast<bf16*>(smraw);  // [2][3 matrices kg, qg, ke][3 terms][16][LD]
  bf16* Vs = Tl + 18 * TILE;                  // [2][16][LV]
  float* Ge = reinterpret_cast<float*>(Vs + 2 * 16 * LV);  // [2][DIM] decay of the whole block
  const int hk = h / (H / a.G), v_base = blockIdx.x * 64, vcol = v_base + warp * 16 + gq;
  const bf16* q = static_cast<const bf16*>(a.q) + (long long)hk * dim;
  const bf16* k = static_cast<const bf16*>(a.k) + (long long)hk * dim;
  const bf16* vp = static_cast<const bf16*>(a.v) + (long long)h * vdim + v_base;
  const float* lgp = a.decay + (long long)h * dim;
  float* stp = a.state + (((long long)a.entry_slot[e] * H + h) * dim) * vdim;
  float S[DIM / 8][4];
  load_state<DIM>(S, stp, dim, vdim, vcol, tq, a.entry_ctx[e] == 0);
  const int r = tid >> 3, c8 = tid & 7;  // this thread's token row and first group of 8 channels of a tile
  uint4 rk[NI], rq[NI];
  float4 rl[NI][2], re[NI][2];
  float ik = 0.f, iq = 0.f;
  auto fetch_raw = [&](int t0) {
    const int t = t0 + r;
    const bool row_ok = t < n;
    const long long row = row0 + t, last = row0 + min(n, t0 + 16) - 1;
    ik = row_ok ? a.inv[row * a.ldi + a.G + hk] : 0.f;
    iq = row_ok ? a.inv[row * a.ldi + hk] : 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = (c8 + 8 * i) * 8;
      const bool col_ok = c < dim, ok = row_ok && col_ok;
      rk[i] = ok ? *reinterpret_cast<const uint4*>(k + row * a.ldk + c) : make_uint4(0, 0, 0, 0);
      rq[i] = ok ? *reinterpret_cast<const uint4*>(q + row * a.ldq + c) : make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        rl[i][x] = ok ? *reinterpret_cast<const float4*>(lgp + row * a.lda + c + 4 * x) : make_float4(0.f, 0.f, 0.f, 0.f);
        re[i][x] = col_ok ? *reinterpret_cast<const float4*>(lgp + last * a.lda + c + 4 * x) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
  };
  auto fetch_v = [&](int t0, int buf) {
    const int c = c8 * 8;
    const bool ok = t0 + r < n && v_base + c < vdim;
    cp_async16(smem_u32(Vs + (buf * 16 + r) * LV + c), vp + (row0 + (ok ? t0 + r : 0)) * a.ldv + (ok ? c : 0), ok);
    pg::cp_async_commit();
  };
  auto form_tiles = [&](int buf) {
    bf16* base = Tl + buf * 9 * TILE + r * LD;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = (c8 + 8 * i) * 8;
      if (c >= DIM) continue;
      const uint32_t kw[4] = {rk[i].x, rk[i].y, rk[i].z, rk[i].w}, qw[4] = {rq[i].x, rq[i].y, rq[i].z, rq[i].w};
      const float l[8] = {rl[i][0].x, rl[i][0].y, rl[i][0].z, rl[i][0].w, rl[i][1].x, rl[i][1].y, rl[i][1].z, rl[i][1].w};
      const float le[8] = {re[i][0].x, re[i][0].y, re[i][0].z, re[i][0].w, re[i][1].x, re[i][1].y, re[i][1].z, re[i][1].w};
      uint32_t t[9][4];
#pragma unroll
      for (int p = 0; p < 4; ++p) {
        const float f0 = exp2f(l[2 * p]), f1 = exp2f(l[2 * p + 1]);
        const float k0 = lo_f(kw[p]) * ik, k1 = hi_f(kw[p]) * ik;
        cut3(k0 * f0, k1 * f1, t[0][p], t[1][p], t[2][p]);
        cut3(lo_f(qw[p]) * iq * f0, hi_f(qw[p]) * iq * f1, t[3][p], t[4][p], t[5][p]);
        // a row past the end has k = 0; its exponent must only not overflow
        cut3(k0 * exp2f(fminf(le[2 * p] - l[2 * p], 0.f)), k1 * exp2f(fminf(le[2 * p + 1] - l[2 * p + 1], 0.f)), t[6][p], t[7][p], t[8][p]);
      }
#pragma unroll
      for (int m = 0; m < 9; ++m) *reinterpret_cast<uint4*>(base + m * TILE + c) = make_uint4(t[m][0], t[m][1], t[m][2], t[m][3]);
      if (r == 0) {
#pragma unroll
        for (int x = 0; x < 8; ++x) Ge[buf * DIM + c + x] = exp2f(le[x]);
      }
    }
  };
  const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = ((lane >> 4) & 1) * 8;
  const int b_row = (lane & 7) + ((lane >> 4) & 1) * 8, b_col = ((lane >> 3) & 1) * 8;
  const uint4* frag = scratch + (block_index(a, e, 0) * H + h) * 6 * 32 + lane;
  const long long frag_step = (long long)H * 6 * 32;
  uint4 fw[3], fb[3];
  fetch_raw(0);
  fetch_v(0, 0);
#pragma unroll
  for (int x = 0; x < 3; ++x) { fw[x] = frag[x * 32]; fb[x] = frag[(3 + x) * 32]; }
  form_tiles(0);
  if (16 < n) fetch_raw(16);
  int cur = 0;
  for (int t0 = 0; t0 < n; t0 += 16, cur ^= 1) {
    pg::cp_async_wait<0>();
    __syncthreads();  // this block's tiles are complete; every warp is done with the other buffers
    const bool more = t0 + 16 < n;
    if (more) {
      fetch_v(t0 + 16, cur ^ 1);
      form_tiles(cur ^ 1);
      if (t0 + 32 < n) fetch_raw(t0 + 32);
    }
    const bf16* kg = Tl + cur * 9 * TILE;
    const bf16* qg = kg + 3 * TILE;
    const bf16* ke = qg + 3 * TILE;
    float xx[4][4] = {};  // (kg S)^T of the two halves of the block, then (qg S)^T
#pragma unroll
    for (int kd = 0; kd < DIM / 16; ++kd) {
      uint32_t sa[3][4], b0[4][3], b1[4][3];
      cut_tiles(S[2 * kd], S[2 * kd + 1], sa);
#pragma unroll
      for (int x = 0; x < 3; ++x) {
        ldmatrix_x4(smem_u32(kg + x * TILE + b_row * LD + kd * 16 + b_col), b0[0][x], b1[0][x], b0[1][x], b1[1][x]);
        ldmatrix_x4(smem_u32(qg + x * TILE + b_row * LD + kd * 16 + b_col), b0[2][x], b1[2][x], b0[3][x], b1[3][x]);
      }
      mma6<4>(xx, sa, b0, b1);
    }
    // R^T = V^T - (kg S)^T, U^T = R^T W^T
    uint32_t va[4], ra[3][4];
    ldmatrix_x4_trans(smem_u32(Vs + (cur * 16 + b_row) * LV + warp * 16 + b_col), va[0], va[1], va[2], va[3]);
    float u[2][4];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
      u[nb][0] = lo_f(va[2 * nb]) - xx[nb][0]; u[nb][1] = hi_f(va[2 * nb]) - xx[nb][1];
      u[nb][2] = lo_f(va[2 * nb + 1]) - xx[nb][2]; u[nb][3] = hi_f(va[2 * nb + 1]) - xx[nb][3];
    }
    cut_tiles(u[0], u[1], ra);
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) u[nb][0] = u[nb][1] = u[nb][2] = u[nb][3] = 0.f;
    mma6_pair(u, ra, fw);
    cut_tiles(u[0], u[1], ra);
    float y[2][4];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) { y[nb][0] = xx[2 + nb][0]; y[nb][1] = xx[2 + nb][1]; y[nb][2] = xx[2 + nb][2]; y[nb][3] = xx[2 + nb][3]; }
    mma6_pair(y, ra, fb);
    if (more) {
      frag += frag_step;
#pragma unroll
      for (int x = 0; x < 3; ++x) { fw[x] = frag[x * 32]; fb[x] = frag[(3 + x) * 32]; }
    }
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = t0 + nb * 8 + 2 * tq + (i & 1), c = vcol + (i >> 1) * 8;
        if (t < n && c < vdim) a.out[(row0 + t) * ((long long)H * vdim) + (long long)h * vdim + c] = y[nb][i];
      }
#pragma unroll
    for (int dp = 0; dp < DIM / 32; ++dp) {
      uint32_t b0[4][3], b1[4][3];
#pragma unroll
      for (int x = 0; x < 3; ++x)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf)
          ldmatrix_x4_trans(smem_u32(ke + x * TILE + a_row * LD + (2 * dp + hf) * 16 + a_col), b0[2 * hf][x], b1[2 * hf][x], b0[2 * hf + 1][x], b1[2 * hf + 1][x]);
      float acc[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 g = *reinterpret_cast<const float2*>(Ge + cur * DIM + dp * 32 + i * 8 + 2 * tq);
        const float(&st)[4] = S[4 * dp + i];
        acc[i][0] = st[0] * g.x; acc[i][1] = st[1] * g.y; acc[i][2] = st[2] * g.x; acc[i][3] = st[3] * g.y;
      }
      mma6<4>(acc, ra, b0, b1);
#pragma unroll
      for (int i = 0; i < 4; ++i) { S[4 * dp + i][0] = acc[i][0]; S[4 * dp + i][1] = acc[i][1]; S[4 * dp + i][2] = acc[i][2]; S[4 * dp + i][3] = acc[i][3]; }
    }
  }
  store_state<DIM>(S, stp, dim, vdim, vcol, tq);
}

inline bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename K>
int set_smem(K kern, size_t smem) {
  if (smem > 220 * 1024) return PG_ERR_ARG;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return PG_ERR_CUDA;
  return PG_OK;
}

template <int DIM, int C, int KIND>
int launch_gated(const PgGatedArgs& a, int n_min, cudaStream_t st) {
  const size_t smem = (size_t)(2 * (2 * C * (DIM + 8) + C * 72) + 3 * C * (C + 8)) * sizeof(bf16) + (size_t)(2 * 5 * C + 4 + 3 * C + DIM) * sizeof(float);
  auto kern = gated_block_kernel<DIM, C, KIND>;
  const int rc = set_smem(kern, smem);
  if (rc != PG_OK) return rc;
  kern<<<dim3((a.vdim + 63) / 64, a.H, a.entries), 128, smem, st>>>(a, n_min);
  pg_count_launch(1);
  return cudaGetLastError() == cudaSuccess ? PG_OK : PG_ERR_CUDA;
}

template <int DIM>
int launch_delta(const PgDeltaArgs& a, float* decay, uint4* scratch, int max_n, int n_min, cudaStream_t st) {
  constexpr int DP = (DIM + 31) / 32 * 32;
  const size_t s1 = (size_t)(72 * (DP + 4) + 3 * 16 * 17 + 48) * sizeof(float);
  auto k1 = delta_blocks_kernel<DP>;
  int rc = set_smem(k1, s1);
  if (rc != PG_OK) return rc;
  k1<<<dim3((max_n + 15) / 16, a.H, a.entries), 128, s1, st>>>(a, decay, scratch, n_min);
  pg_count_launch(1);
  const size_t s2 = (size_t)(18 * 16 * (DIM + 8) + 2 * 16 * 72) * sizeof(bf16) + (size_t)2 * DIM * sizeof(float);
  auto k2 = delta_chain_kernel<DIM>;
  rc = set_smem(k2, s2);
  if (rc != PG_OK) return rc;
  k2<<<dim3((a.vdim + 63) / 64, a.H, a.entries), 128, s2, st>>>(a, scratch, n_min);
  pg_count_launch(1);
  return cudaGetLastError() == cudaSuccess ? PG_OK : PG_ERR_CUDA;
}

}  // namespace

extern "C" int pg_gated_blocks(const PgGatedArgs* a, int kind, int n_min, void* stream) {
  if (a == nullptr || a->entries <= 0 || a->entries > 65535 || a->H <= 0 || a->H > 65535 || a->G <= 0 || a->H % a->G || (kind != 0 && kind != 1) ||
      (kind == 1 && (a->norm_state == nullptr || a->gate2 == nullptr || !(a->cap > 0.f))) || (kind == 0 && a->p3 == nullptr))
    return PG_ERR_ARG;
  // 16-byte row fetches
  if (a->dim <= 0 || a->dim % 8 || a->dim > 128 || a->vdim <= 0 || a->vdim % 8 || a->ldq % 8 || a->ldk % 8 || a->ldv % 8 || !al16(a->q) || !al16(a->k) || !al16(a->v))
    return PG_ERR_ARG;
  cudaStream_t st = PG_ST(stream);
#define PG_GB(D, C) return kind == 0 ? launch_gated<D, C, 0>(*a, n_min, st) : launch_gated<D, C, 1>(*a, n_min, st)
  if (a->dim <= 32) PG_GB(32, 64);
  if (a->dim <= 64) PG_GB(64, 64);
  if (a->dim <= 96) PG_GB(96, 32);
  PG_GB(128, 32);
#undef PG_GB
}

extern "C" int pg_delta_blocks(const PgDeltaArgs* a, float* decay, void* scratch, int max_n, int n_min, void* stream) {
  if (a == nullptr || a->entries <= 0 || a->entries > 65535 || a->H <= 0 || a->H > 65535 || a->G <= 0 || a->H % a->G || scratch == nullptr || max_n <= 0 ||
      decay != a->decay)
    return PG_ERR_ARG;
  if (a->dim <= 0 || a->dim % 8 || a->dim > 128 || a->vdim <= 0 || a->vdim % 8 || a->ldq % 8 || a->ldk % 8 || a->ldv % 8 || a->lda % 4 || !al16(a->q) || !al16(a->k) ||
      !al16(a->v) || !al16(decay) || !al16(scratch))
    return PG_ERR_ARG;
  cudaStream_t st = PG_ST(stream);
  uint4* sc = static_cast<uint4*>(scratch);
  if (a->dim <= 32) return launch_delta<32>(*a, decay, sc, max_n, n_min, st);
  if (a->dim <= 64) return launch_delta<64>(*a, decay, sc, max_n, n_min, st);
  if (a->dim <= 96) return launch_delta<96>(*a, decay, sc, max_n, n_min, st);
  return launch_delta<128>(*a, decay, sc, max_n, n_min, st);
}
