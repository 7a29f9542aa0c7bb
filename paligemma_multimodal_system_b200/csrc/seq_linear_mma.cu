// Decayed linear attention of prompt portions in bf16 on the tensor cores (the block form of pg_linear_attn_scan for layers without silu),
// with every quantity of the recurrence at fp32 precision: queries and keys are turned and scaled in fp32 as they are staged and enter
// the products as three bf16 terms (8 + 8 + 8 mantissa bits), as do the state and the decay-weighted scores and values.
//
// With a = decay, block rows i, j = 0 .. c-1 and S the state before the block:
//   o_i = a^(i+1) S^T q_i + sum_{j <= i} P_ij v_j,  P_ij = a^(i-j) (q_i . k_j);      S' = a^c S + sum_j a^(c-1-j) k_j v_j^T
//
// A CTA advances 64 value columns of one head of one entry through all its new tokens.  The state is held TRANSPOSED, S^T [value column, key
// dimension], as the fp32 accumulators of m16n8k16 tiles (warp = 16 value columns): two adjacent 8-column accumulator tiles are, element
// for element, the A operand of a 16-deep product step.  The raw rows of the next block and its cosines / sines are fetched into registers,
// its values with cp.async, while the current block is multiplied.
#include "common.cuh"
#include "paligemma_b200.h"

using bf16 = __nv_bfloat16;
using pg::cp_async16;
using pg::ldmatrix_x4;
using pg::ldmatrix_x4_trans;
using pg::mma_bf16_16816;
using pg::smem_u32;

namespace {

__device__ __forceinline__ float lo_f(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float hi_f(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }

// (p, q) = sum of three bf16 pairs, packed
__device__ __forceinline__ void cut3(float p, float q, uint32_t& a, uint32_t& b, uint32_t& c) {
  a = pg::pack_bf16(p, q);
  const float p1 = p - lo_f(a), q1 = q - hi_f(a);
  b = pg::pack_bf16(p1, q1);
  c = pg::pack_bf16(p1 - lo_f(b), q1 - hi_f(b));
}

template <int DIM, int C>
__global__ void __launch_bounds__(128, 2) linear_attn_block_kernel(const bf16* __restrict__ qkv, long long ld, float* __restrict__ state,
                                                                   const float* __restrict__ decay, float* __restrict__ out,
                                                                   const int* __restrict__ entry_row0, const int* __restrict__ entry_n,
                                                                   const int* __restrict__ entry_ctx, const int* __restrict__ entry_slot, int H, int dim,
                                                                   int vdim, PgLinearAttnOps ops) {
  constexpr int LD = DIM + 8, LV = 64 + 8, LP = C + 8, CH = DIM / 8, NI = C * CH / 128, TILE = C * LD, R = C / 16;
  static_assert(C * CH % 128 == 0, "every thread stages the same number of 8-element pieces");
  const int e = blockIdx.z, h = blockIdx.y;
  const int n = entry_n[e];
  if (n < ops.n_min || n > ops.n_max) return;
  const long long row0 = entry_row0[e];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, tq = lane & 3;
  extern __shared__ __align__(16) unsigned char smraw[];
  bf16* Qs = reinterpret_cast<bf16*>(smraw);  // [3 terms][C][LD]
  bf16* Ks = Qs + 3 * TILE;                   // [3 terms][C][LD]
  bf16* Ps = Ks + 3 * TILE;                   // [3 terms][C][LP]
  bf16* Vs = Ps + 3 * C * LP;                 // [2][C][LV]
  float* ap = reinterpret_cast<float*>(Vs + 2 * C * LV);  // a^0 .. a^C
  const int v_base = blockIdx.x * 64, vcol = v_base + warp * 16 + gq;
  const bf16* qp = qkv + (long long)h * dim;
  const bf16* kp = qkv + (long long)(H + h) * dim;
  const bf16* vp = qkv + 2LL * H * dim + (long long)h * vdim + v_base;
  float* stp = state + (((long long)entry_slot[e] * H + h) * dim) * vdim;
  const bool fresh = entry_ctx[e] == 0;
  float S[DIM / 8][4];
#pragma unroll
  for (int nb = 0; nb < DIM / 8; ++nb)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = nb * 8 + 2 * tq + (i & 1), c = vcol + (i >> 1) * 8;
      S[nb][i] = (!fresh && d < dim && c < vdim) ? stp[(long long)d * vdim + c] : 0.f;
    }
  for (int i = tid; i <= C; i += 128) ap[i] = (float)pow((double)decay[h], (double)i);
  uint4 rq[NI], rk[NI];
  float4 rc[NI], rs[NI];
  auto fetch = [&](int t0, int buf) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int id = tid + 128 * i, r = id / CH, c = (id % CH) * 8;
      const bool ok = t0 + r < n && c < dim;
      const long long row = row0 + t0 + r;
      rq[i] = ok ? *reinterpret_cast<const uint4*>(qp + row * ld + c) : make_uint4(0, 0, 0, 0);
      rk[i] = ok ? *reinterpret_cast<const uint4*>(kp + row * ld + c) : make_uint4(0, 0, 0, 0);
      const bool turn = ok && ops.rotate != nullptr;
      rc[i] = turn ? *reinterpret_cast<const float4*>(ops.rotate + row * 2 * ops.pairs + c / 2) : make_float4(1.f, 1.f, 1.f, 1.f);
      rs[i] = turn ? *reinterpret_cast<const float4*>(ops.rotate + (row * 2 + 1) * ops.pairs + c / 2) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int id = tid; id < C * 8; id += 128) {
      const int r = id / 8, c = (id % 8) * 8;
      const bool ok = t0 + r < n && v_base + c < vdim;
      cp_async16(smem_u32(Vs + (buf * C + r) * LV + c), vp + (row0 + (ok ? t0 + r : 0)) * ld + (ok ? c : 0), ok);
    }
    pg::cp_async_commit();
  };
  auto form_tiles = [&]() {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int id = tid + 128 * i, r = id / CH, c = (id % CH) * 8;
      const uint32_t qw[4] = {rq[i].x, rq[i].y, rq[i].z, rq[i].w}, kw[4] = {rk[i].x, rk[i].y, rk[i].z, rk[i].w};
      const float cs[4] = {rc[i].x, rc[i].y, rc[i].z, rc[i].w}, sn[4] = {rs[i].x, rs[i].y, rs[i].z, rs[i].w};
      uint32_t t[6][4];
#pragma unroll
      for (int p = 0; p < 4; ++p) {
        const float q0 = lo_f(qw[p]), q1 = hi_f(qw[p]), k0 = lo_f(kw[p]), k1 = hi_f(kw[p]);
        cut3(q0 * cs[p] - q1 * sn[p], q1 * cs[p] + q0 * sn[p], t[0][p], t[1][p], t[2][p]);
        cut3((k0 * cs[p] - k1 * sn[p]) * ops.kscale, (k1 * cs[p] + k0 * sn[p]) * ops.kscale, t[3][p], t[4][p], t[5][p]);
      }
      bf16* to = Qs + r * LD + c;  // Ks follows Qs: six tiles one after the other
#pragma unroll
      for (int m = 0; m < 6; ++m) *reinterpret_cast<uint4*>(to + m * TILE) = make_uint4(t[m][0], t[m][1], t[m][2], t[m][3]);
    }
  };
  // lane's row / column inside a 16 x 16 block for ldmatrix: A operand (row-major), B operand (rows = n), and their transposed forms
  const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = ((lane >> 4) & 1) * 8;
  const int b_row = (lane & 7) + ((lane >> 4) & 1) * 8, b_col = ((lane >> 3) & 1) * 8;
  fetch(0, 0);
  int cur = 0;
  for (int t0 = 0; t0 < n; t0 += C, cur ^= 1) {
    const int cn = min(C, n - t0);
    form_tiles();
    pg::cp_async_wait<0>();
    __syncthreads();  // this block's tiles are there
    if (t0 + C < n) fetch(t0 + C, cur ^ 1);
    const bf16* Vb = Vs + cur * C * LV;
    // P: the 16 x 16 blocks on and below the diagonal, shared out over the warps
    for (int id = warp; id < R * (R + 1) / 2; id += 4) {
      int ib = 0, jb = id;
      while (jb > ib) { jb -= ib + 1; ++ib; }
      float s[2][4] = {}, s2[2][4] = {};
#pragma unroll
      for (int kd = 0; kd < DIM / 16; ++kd) {
        uint32_t qa[3][4], kb[3][4];
#pragma unroll
        for (int x = 0; x < 3; ++x) {
          ldmatrix_x4(smem_u32(Qs + x * TILE + (ib * 16 + a_row) * LD + kd * 16 + a_col), qa[x][0], qa[x][1], qa[x][2], qa[x][3]);
          ldmatrix_x4(smem_u32(Ks + x * TILE + (jb * 16 + b_row) * LD + kd * 16 + b_col), kb[x][0], kb[x][1], kb[x][2], kb[x][3]);
        }
#pragma unroll
        for (int x = 0; x < 6; ++x) {  // two operands in three terms each (dropped products lie below 2^-24), four chains of accumulators
          constexpr int TERM_A[6] = {0, 0, 1, 1, 0, 2}, TERM_B[6] = {0, 1, 0, 1, 2, 0};
          float(&to)[2][4] = (x & 1) ? s2 : s;
          mma_bf16_16816(to[0], qa[TERM_A[x]], kb[TERM_B[x]][0], kb[TERM_B[x]][1]);
          mma_bf16_16816(to[1], qa[TERM_A[x]], kb[TERM_B[x]][2], kb[TERM_B[x]][3]);
        }
      }
      const int tl = ib * 16 + gq, th = tl + 8;
#pragma unroll
      for (int nb = 0; nb < 2; ++nb) {
        const int j = jb * 16 + nb * 8 + 2 * tq;
        float p[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int away = ((i & 2) ? th : tl) - (j + (i & 1));
          p[i] = away >= 0 ? (s[nb][i] + s2[nb][i]) * ap[away >= 0 ? away : 0] : 0.f;
        }
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
    // outputs O^T [16 value columns, C tokens]: the part of the carried state (needs no P)
    float o[C / 8][4];
#pragma unroll
    for (int i = 0; i < C / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    if (!(fresh && t0 == 0)) {
#pragma unroll
      for (int kd = 0; kd < DIM / 16; ++kd) {
        uint32_t sa[3][4];
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          cut3(S[2 * kd + hf][0], S[2 * kd + hf][1], sa[0][2 * hf], sa[1][2 * hf], sa[2][2 * hf]);
          cut3(S[2 * kd + hf][2], S[2 * kd + hf][3], sa[0][2 * hf + 1], sa[1][2 * hf + 1], sa[2][2 * hf + 1]);
        }
#pragma unroll
        for (int y = 0; y < 3; ++y) {
          uint32_t bq[R][4];
#pragma unroll
          for (int tb = 0; tb < R; ++tb)
            ldmatrix_x4(smem_u32(Qs + y * TILE + (tb * 16 + b_row) * LD + kd * 16 + b_col), bq[tb][0], bq[tb][1], bq[tb][2], bq[tb][3]);
#pragma unroll
          for (int x = 0; x < 3 - y; ++x)  // terms (0,0) (1,0) (2,0) (0,1) (1,1) (0,2)
#pragma unroll
            for (int tb = 0; tb < R; ++tb) {
              mma_bf16_16816(o[2 * tb], sa[x], bq[tb][0], bq[tb][1]);
              mma_bf16_16816(o[2 * tb + 1], sa[x], bq[tb][2], bq[tb][3]);
            }
        }
      }
#pragma unroll
      for (int nb = 0; nb < C / 8; ++nb) {
        const float c0 = ap[nb * 8 + 2 * tq + 1], c1 = ap[nb * 8 + 2 * tq + 2];
        o[nb][0] *= c0; o[nb][1] *= c1; o[nb][2] *= c0; o[nb][3] *= c1;
      }
    }
    const float carry = ap[cn];
#pragma unroll
    for (int nb = 0; nb < DIM / 8; ++nb) { S[nb][0] *= carry; S[nb][1] *= carry; S[nb][2] *= carry; S[nb][3] *= carry; }
    __syncthreads();  // P is complete
#pragma unroll
    for (int kk = 0; kk < R; ++kk) {
      uint32_t va[4], wa[3][4];
      ldmatrix_x4_trans(smem_u32(Vb + (kk * 16 + b_row) * LV + warp * 16 + b_col), va[0], va[1], va[2], va[3]);
#pragma unroll
      for (int x = 0; x < 3; ++x)
#pragma unroll
        for (int tb = kk; tb < R; ++tb) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(smem_u32(Ps + (x * C + tb * 16 + b_row) * LP + kk * 16 + b_col), b0, b1, b2, b3);
          mma_bf16_16816(o[2 * tb], va, b0, b1);
          mma_bf16_16816(o[2 * tb + 1], va, b2, b3);
        }
      // state: values weighted by a^(c-1-j) against the keys
      const int j = kk * 16 + 2 * tq;
      auto weight = [&](int t) { return t < cn ? ap[cn - 1 - t] : 0.f; };
      const float w0 = weight(j), w1 = weight(j + 1), w2 = weight(j + 8), w3 = weight(j + 9);
      cut3(lo_f(va[0]) * w0, hi_f(va[0]) * w1, wa[0][0], wa[1][0], wa[2][0]);
      cut3(lo_f(va[1]) * w0, hi_f(va[1]) * w1, wa[0][1], wa[1][1], wa[2][1]);
      cut3(lo_f(va[2]) * w2, hi_f(va[2]) * w3, wa[0][2], wa[1][2], wa[2][2]);
      cut3(lo_f(va[3]) * w2, hi_f(va[3]) * w3, wa[0][3], wa[1][3], wa[2][3]);
#pragma unroll
      for (int y = 0; y < 3; ++y)
#pragma unroll
        for (int dp = 0; dp < DIM / 32; ++dp) {
          uint32_t bk[2][4];
#pragma unroll
          for (int hf = 0; hf < 2; ++hf)
            ldmatrix_x4_trans(smem_u32(Ks + y * TILE + (kk * 16 + a_row) * LD + (2 * dp + hf) * 16 + a_col), bk[hf][0], bk[hf][1], bk[hf][2], bk[hf][3]);
#pragma unroll
          for (int x = 0; x < 3 - y; ++x)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
              mma_bf16_16816(S[4 * dp + 2 * hf], wa[x], bk[hf][0], bk[hf][1]);
              mma_bf16_16816(S[4 * dp + 2 * hf + 1], wa[x], bk[hf][2], bk[hf][3]);
            }
        }
    }
#pragma unroll
    for (int nb = 0; nb < C / 8; ++nb)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = nb * 8 + 2 * tq + (i & 1), c = vcol + (i >> 1) * 8;
        if (t < cn && c < vdim) out[(row0 + t0 + t) * ((long long)H * vdim) + (long long)h * vdim + c] = o[nb][i];
      }
    __syncthreads();  // every warp is done with the tiles before the next block's are formed
  }
#pragma unroll
  for (int nb = 0; nb < DIM / 8; ++nb)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = nb * 8 + 2 * tq + (i & 1), c = vcol + (i >> 1) * 8;
      if (d < dim && c < vdim) stp[(long long)d * vdim + c] = S[nb][i];
    }
}

template <int DIM, int C>
int launch_blocks(const bf16* qkv, long long ld, float* state, const float* decay, float* out, const int* row0, const int* n, const int* ctx,
                  const int* slot, int entries, int H, int dim, int vdim, const PgLinearAttnOps& ops, cudaStream_t st) {
  const size_t smem = (size_t)(6 * C * (DIM + 8) + 3 * C * (C + 8) + 2 * C * 72) * sizeof(bf16) + (C + 1) * sizeof(float);
  auto kern = linear_attn_block_kernel<DIM, C>;
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return PG_ERR_CUDA;
  kern<<<dim3((vdim + 63) / 64, H, entries), 128, smem, st>>>(qkv, ld, state, decay, out, row0, n, ctx, slot, H, dim, vdim, ops);
  pg_count_launch(1);
  return cudaGetLastError() == cudaSuccess ? PG_OK : PG_ERR_CUDA;
}

}  // namespace

extern "C" int pg_linear_attn_blocks(const void* qkv, long long ld, float* state, const float* decay, float* out, const int* entry_row0,
                                     const int* entry_n, const int* entry_ctx, const int* entry_slot, int entries, int H, int dim, int vdim,
                                     const PgLinearAttnOps* options, void* stream) {
  if (entries <= 0 || entries > 65535 || H <= 0 || H > 65535 || options == nullptr || options->silu) return PG_ERR_ARG;
  // 16-byte fetches of the rows, of the cosines and of the sines
  if (dim <= 0 || dim % 8 || dim > 128 || vdim <= 0 || vdim % 8 || ld % 8 || (reinterpret_cast<uintptr_t>(qkv) & 15)) return PG_ERR_ARG;
  if (options->rotate != nullptr && (2 * options->pairs < dim || options->pairs % 4 || (reinterpret_cast<uintptr_t>(options->rotate) & 15))) return PG_ERR_ARG;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
#define PG_LB(D, C) \
  return launch_blocks<D, C>(static_cast<const bf16*>(qkv), ld, state, decay, out, entry_row0, entry_n, entry_ctx, entry_slot, entries, H, dim, vdim, *options, st)
  if (dim <= 32) PG_LB(32, 64);
  if (dim <= 64) PG_LB(64, 64);
  if (dim <= 96) PG_LB(96, 32);
  PG_LB(128, 32);
#undef PG_LB
}
