// retention.cu — retention: linear attention with a constant decay per head over rotated queries and keys,
//     S <- lambda_h S + k v^T,   o = S^T q,   out = o / sqrt(mean(o^2) + eps) * silu(gate)
// with k times dim^-1/2, per head an fp32 state S [dim][vdim] in the sequence's slot.
//
// Single tokens: one kernel per (sequence, head) turns the vectors, advances the state (one pass over it) and finishes
// the output.  Portions: a preparation turns the vectors of all tokens, then either the token-by-token recurrence of
// decay_attn.cu (fp32 models, sizes the tiles do not take) or the chunk kernel below runs, and a last kernel norms and
// gates the outputs.
//
// Chunks of 64 tokens on the tensor cores (bf16 models): with local indices i, j of a chunk of n tokens that starts from S,
//     o_i = lambda^(i+1) S^T q_i + sum_{j <= i} lambda^(i-j) (q_i . k_j) v_j
//     S'  = lambda^n S + sum_j lambda^(n-1-j) k_j v_j^T
// Four small products.  Operands that are not bf16 to begin with (turned q and k, S, decayed v, the weighted scores) enter
// as a bf16 high part plus a bf16 low part, so a product keeps about 16 bits of each factor; sums and S itself are fp32.
#include <math.h>

#include <algorithm>

#include "layered_common.cuh"

namespace b200q {

struct SeqView {
  int row0, n, pos0, slot;
};
__device__ __forceinline__ SeqView seq_view(const int32_t* __restrict__ seq_desc, int s) {
  const int4 v = *reinterpret_cast<const int4*>(seq_desc + 4 * s);
  return {v.x, v.y, v.z, v.w};
}
__device__ __forceinline__ void cp_async16(void* smem_dst, const void* gsrc) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem_dst)), "l"(gsrc) : "memory");
}

// value d of a head's vector v, turned by the token's row `cs` of cosines and sines
template <typename T>
__device__ __forceinline__ float turned(const T* v, int d, int half, const float2* cs) {
  if (d >= 2 * half) return ldf(v + d);
  const int i = d < half ? d : d - half;
  const float a = ldf(v + i), b = ldf(v + i + half);
  const float2 t = cs[i];
  return d < half ? a * t.x - b * t.y : b * t.x + a * t.y;
}

// ------------------------------------------------------------------------------------------------
// single tokens: CTA per (sequence, head).  The state is walked once, V columns per thread; a thread keeps its columns
// and takes every `groups`-th row, loads of RET_ROWS rows in flight.
// ------------------------------------------------------------------------------------------------
constexpr int RET_THREADS = 256, RET_ROWS = 8;
template <typename T, int V>
__global__ void __launch_bounds__(RET_THREADS) retention_decode_kernel(
    const T* __restrict__ proj, int ldp, int heads, int dim, int vdim, int half, const float2* __restrict__ table,
    const float* __restrict__ decay, float* __restrict__ state, long long slot_stride, const int32_t* __restrict__ seq_desc,
    float eps, T* __restrict__ out) {
  extern __shared__ float sm[];  // q [dim] | k [dim] | partial outputs [groups][vdim]
  __shared__ float red[32];
  const SeqView s = seq_view(seq_desc, blockIdx.x);
  if (s.n != 1) return;  // portions take the other kernels
  const int h = blockIdx.y, tid = threadIdx.x, HD = heads * dim, HV = heads * vdim;
  const long long t = s.row0;
  const T* pr = proj + t * ldp;
  const float2* cs = table + t * half;
  float *qs = sm, *ks = sm + dim, *part = sm + 2 * dim;
  const float kmul = 1.f / sqrtf((float)dim), lam = decay[h];
  const int nc = vdim / V, groups = nc < RET_THREADS ? RET_THREADS / nc : 1;
  const int grp = nc < RET_THREADS ? tid / nc : 0, cv0 = nc < RET_THREADS ? tid % nc : tid;
  float* st = state + (long long)s.slot * slot_stride + (long long)h * dim * vdim;
  float S[RET_ROWS][V];
  auto fetch = [&](int d0, int c) {
#pragma unroll
    for (int r = 0; r < RET_ROWS; ++r) {
      const int d = d0 + r * groups;
      const bool on = d < dim && s.pos0 > 0;  // a sequence that starts here starts from zeros whatever the slot holds
      if constexpr (V == 4) {
        const float4 f = on ? *reinterpret_cast<const float4*>(st + (long long)d * vdim + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[r][0] = f.x; S[r][1] = f.y; S[r][2] = f.z; S[r][3] = f.w;
      } else {
        S[r][0] = on ? st[(long long)d * vdim + c] : 0.f;
      }
    }
  };
  if (grp < groups && cv0 < nc) fetch(grp, cv0 * V);  // on its way while the vectors are turned
  for (int d = tid; d < dim; d += RET_THREADS) {
    qs[d] = turned(pr + h * dim, d, half, cs);
    ks[d] = turned(pr + HD + h * dim, d, half, cs) * kmul;
  }
  __syncthreads();
  if (grp < groups)
    for (int cv = cv0; cv < nc; cv += RET_THREADS) {
      const int c = cv * V;
      float v[V], o[V];
#pragma unroll
      for (int i = 0; i < V; ++i) {
        v[i] = ldf(pr + 2 * HD + h * vdim + c + i);
        o[i] = 0.f;
      }
      for (int d0 = grp; d0 < dim; d0 += groups * RET_ROWS) {
        if (d0 != grp || cv != cv0) fetch(d0, c);
#pragma unroll
        for (int r = 0; r < RET_ROWS; ++r) {
          const int d = d0 + r * groups;
          if (d >= dim) break;
          const float k = ks[d], q = qs[d];
#pragma unroll
          for (int i = 0; i < V; ++i) {
            S[r][i] = fmaf(lam, S[r][i], k * v[i]);
            o[i] = fmaf(S[r][i], q, o[i]);
          }
          float* dst = st + (long long)d * vdim + c;
          if constexpr (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
          else dst[0] = S[r][0];
        }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) part[(long long)grp * vdim + c + i] = o[i];
    }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < vdim; c += RET_THREADS) {  // the groups' parts in a fixed order; each thread its own columns
    float o = part[c];
    for (int g = 1; g < groups; ++g) o += part[(long long)g * vdim + c];
    part[c] = o;
    ss = fmaf(o, o, ss);
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)vdim + eps);
  const T* gate = pr + 2 * HD + HV + h * vdim;
  for (int c = tid; c < vdim; c += RET_THREADS) stf(out + t * HV + h * vdim + c, part[c] * inv * siluf_(ldf(gate + c)));
}

// ------------------------------------------------------------------------------------------------
// preparation for the recurrence: fp32 rows [q | k | v]
// ------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) retention_prep_kernel(const T* __restrict__ proj, int ldp, int heads, int dim, int vdim,
                                                             int half, const float2* __restrict__ table,
                                                             float* __restrict__ qkv) {
  const long long t = blockIdx.x;
  const int HD = heads * dim, HV = heads * vdim;
  const T* pr = proj + t * ldp;
  const float2* cs = table + t * half;
  const float kmul = 1.f / sqrtf((float)dim);
  float* o = qkv + t * (2 * HD + HV);
  for (int e = threadIdx.x; e < 2 * HD; e += blockDim.x)
    o[e] = turned(pr + (e / dim) * dim, e % dim, half, cs) * (e < HD ? 1.f : kmul);
  for (int e = threadIdx.x; e < HV; e += blockDim.x) o[2 * HD + e] = ldf(pr + 2 * HD + e);
}

__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  lo = pack_bf16x2(a - bf16_lo(hi), b - bf16_hi(hi));
}

// preparation for the chunk kernel: bf16 rows [q high | q low | k high | k low].  A thread takes 8 neighbouring values of a
// head (and their 8 partners where they turn); half is a multiple of 8.
__global__ void __launch_bounds__(256) retention_split_kernel(const bf16* __restrict__ proj, int ldp, int heads, int dim,
                                                              int half, const float2* __restrict__ table,
                                                              bf16* __restrict__ qk, long long total) {
  const int HD = heads * dim, per_head = dim / 8 - half / 8, per = 2 * heads * per_head;
  const float kmul = 1.f / sqrtf((float)dim);
  for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
    const long long t = e / per;
    const int r = (int)(e - t * per), vec = r / per_head, piece = r - vec * per_head;  // vec: q heads, then k heads
    const bool pair = piece < half / 8;
    const int d = pair ? piece * 8 : half + piece * 8;  // unturned pieces follow the turned 2 * half values
    const float mul = vec < heads ? 1.f : kmul;
    const bf16* src = proj + t * ldp + (long long)vec * dim + d;
    bf16* dst = qk + t * 4 * HD + (vec < heads ? (long long)vec * dim : 2ll * HD + (long long)(vec - heads) * dim) + d;
    const uint4 a4 = ld_v4(src);
    const uint32_t aw[4] = {a4.x, a4.y, a4.z, a4.w};
    float a[8], b[8];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      a[2 * i] = bf16_lo(aw[i]);
      a[2 * i + 1] = bf16_hi(aw[i]);
    }
    if (pair) {
      const uint4 b4 = ld_v4(src + half);
      const uint32_t bw[4] = {b4.x, b4.y, b4.z, b4.w};
      const float2* cs = table + t * half + d;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float u = a[i], v = i & 1 ? bf16_hi(bw[i / 2]) : bf16_lo(bw[i / 2]);
        const float2 c = cs[i];
        a[i] = u * c.x - v * c.y;
        b[i] = v * c.x + u * c.y;
      }
    }
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) split_pair(a[2 * i] * mul, a[2 * i + 1] * mul, hi[i], lo[i]);
    st_v4(dst, make_uint4(hi[0], hi[1], hi[2], hi[3]));
    st_v4(dst + HD, make_uint4(lo[0], lo[1], lo[2], lo[3]));
    if (pair) {
#pragma unroll
      for (int i = 0; i < 4; ++i) split_pair(b[2 * i] * mul, b[2 * i + 1] * mul, hi[i], lo[i]);
      st_v4(dst + half, make_uint4(hi[0], hi[1], hi[2], hi[3]));
      st_v4(dst + HD + half, make_uint4(lo[0], lo[1], lo[2], lo[3]));
    }
  }
}

// ------------------------------------------------------------------------------------------------
// chunks: CTA of 4 warps per (sequence, head, VB value columns), walking the portion 64 tokens at a time; warp w owns the
// chunk's rows [16w, 16w + 16) and the state's rows [w DT/4, (w + 1) DT/4), which stay in its registers as fp32
// accumulators.  q, k (high and low parts) and v of the next chunk arrive by cp.async while this one is multiplied.
// ------------------------------------------------------------------------------------------------
constexpr int RCH = 64;
template <int DT, int VB>
struct RetentionSmem {
  static constexpr int LDK = DT + 8, LDV = VB + 8;  // padded rows: ldmatrix rows fall on different banks
  static constexpr int STAGE = RCH * (4 * LDK + LDV);  // elements: q high, q low, k high, k low, v
  static constexpr int BYTES = (2 * STAGE + 2 * RCH * LDV + 2 * DT * LDV) * 2 + (RCH + 1) * 4;
};
template <int DT, int VB>
__global__ void __launch_bounds__(128) retention_chunk_kernel(const bf16* __restrict__ qk, const bf16* __restrict__ v,
                                                              int ldv_row, const float* __restrict__ decay,
                                                              float* __restrict__ state, long long slot_stride,
                                                              const int32_t* __restrict__ seq_desc, int heads, int vdim,
                                                              float* __restrict__ raw) {
  using SM = RetentionSmem<DT, VB>;
  constexpr int LDK = SM::LDK, LDV = SM::LDV, MT = DT / 64, NV = VB / 8;
  extern __shared__ __align__(16) uint8_t smraw[];
  bf16* stage = reinterpret_cast<bf16*>(smraw);
  bf16* vs = stage + 2 * SM::STAGE;       // decayed v: [2][64][LDV], high and low parts
  bf16* ss = vs + 2 * RCH * LDV;          // the state before the chunk: [2][DT][LDV], high and low parts
  float* pw = reinterpret_cast<float*>(ss + 2 * DT * LDV);  // lambda^i, i <= 64
  const SeqView s = seq_view(seq_desc, blockIdx.x);
  if (s.n <= 1) return;  // single tokens: the fused kernel's
  const int h = blockIdx.y, v0 = blockIdx.z * VB, HD = heads * DT, HV = heads * vdim;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, q4 = lane & 3;
  const int nchunks = (s.n + RCH - 1) / RCH;
  auto load_chunk = [&](int c, int buf) {
    const int r0 = c * RCH, n = min(RCH, s.n - r0);
    bf16* b = stage + buf * SM::STAGE;
    constexpr int PK = DT / 8, PV = VB / 8, PER = 4 * PK + PV;  // 16-byte pieces of a token
    for (int e = tid; e < RCH * PER; e += 128) {
      const int j = e / PER, p = e % PER;
      const long long row = s.row0 + r0 + j;
      bf16* dst;
      const bf16* src;
      if (p < 4 * PK) {
        const int part = p / PK, d = (p % PK) * 8;
        dst = b + part * RCH * LDK + j * LDK + d;
        src = qk + row * 4 * HD + (long long)part * HD + h * DT + d;
      } else {
        const int d = (p - 4 * PK) * 8;
        dst = b + 4 * RCH * LDK + j * LDV + d;
        src = v + row * ldv_row + (long long)h * vdim + v0 + d;
      }
      if (j < n) cp_async16(dst, src);
      else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load_chunk(0, 0);
  for (int i = tid; i <= RCH; i += 128) pw[i] = (float)pow((double)decay[h], (double)i);
  // this warp's part of the state: rows warp*DT/4 + 16 m + gq (+ 8), columns v0 + 8 n + 2 q4 (+ 1)
  float* st = state + (long long)s.slot * slot_stride + (long long)h * DT * vdim + v0;
  float S[MT][NV][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float* src = st + (long long)(warp * (DT / 4) + m * 16 + gq + 8 * r) * vdim + n * 8 + 2 * q4;
        S[m][n][2 * r] = s.pos0 > 0 ? src[0] : 0.f;
        S[m][n][2 * r + 1] = s.pos0 > 0 ? src[1] : 0.f;
      }
  const uint32_t a_off = (uint32_t)(((warp * 16 + (lane & 15)) * LDK + (lane >> 4) * 8) * 2);  // rows of q
  const uint32_t k_off = (uint32_t)((((lane & 7) + 8 * (lane >> 4)) * LDK + 8 * ((lane >> 3) & 1)) * 2);
  const uint32_t b_off = (uint32_t)(((((lane >> 3) & 1) * 8 + (lane & 7)) * LDV + 8 * (lane >> 4)) * 2);  // [k][n], transposed
  // k as the transposed A operand: entry (d, j) lies at row j, column d
  const uint32_t kt_off = (uint32_t)((((lane & 7) + 8 * (lane >> 4)) * LDK + warp * (DT / 4) + 8 * ((lane >> 3) & 1)) * 2);
  for (int c = 0; c < nchunks; ++c) {
    const int buf = c & 1, n = min(RCH, s.n - c * RCH);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // chunk c has landed; everyone is done with chunk c - 1, with vs and with ss
    if (c + 1 < nchunks) load_chunk(c + 1, buf ^ 1);
    bf16* b = stage + buf * SM::STAGE;
    const bf16* vraw = b + 4 * RCH * LDK;
    for (int e = tid; e < RCH * (VB / 2); e += 128) {
      const int j = e / (VB / 2), d = (e % (VB / 2)) * 2;
      const uint32_t x = *reinterpret_cast<const uint32_t*>(vraw + j * LDV + d);
      const float w = j < n ? pw[n - 1 - j] : 0.f;
      uint32_t hi, lo;
      split_pair(bf16_lo(x) * w, bf16_hi(x) * w, hi, lo);
      *reinterpret_cast<uint32_t*>(vs + j * LDV + d) = hi;
      *reinterpret_cast<uint32_t*>(vs + RCH * LDV + j * LDV + d) = lo;
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int nt = 0; nt < NV; ++nt)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t hi, lo;
          split_pair(S[m][nt][2 * r], S[m][nt][2 * r + 1], hi, lo);
          const int at = (warp * (DT / 4) + m * 16 + gq + 8 * r) * LDV + nt * 8 + 2 * q4;
          *reinterpret_cast<uint32_t*>(ss + at) = hi;
          *reinterpret_cast<uint32_t*>(ss + DT * LDV + at) = lo;
        }
    __syncthreads();
    const uint32_t qh_s = smem_u32(b), ql_s = qh_s + RCH * LDK * 2, kh_s = ql_s + RCH * LDK * 2, kl_s = kh_s + RCH * LDK * 2;
    const uint32_t v_s = kl_s + RCH * LDK * 2, vh_s = smem_u32(vs), vl_s = vh_s + RCH * LDV * 2;
    const uint32_t sh_s = smem_u32(ss), sl_s = sh_s + DT * LDV * 2;
    if (warp * 16 < n) {
      // scores of this warp's 16 tokens against the chunk's keys up to its last token, and S^T q
      float sc[8][4], o[NV][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < DT / 16; ++ks) {
        uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
        ldsm_x4(qh_s + a_off + ks * 32, h0, h1, h2, h3);
        ldsm_x4(ql_s + a_off + ks * 32, l0, l1, l2, l3);
#pragma unroll
        for (int nt2 = 0; nt2 < 4; ++nt2) {
          if (nt2 > warp) break;
          uint32_t b0, b1, b2, b3, c0, c1, c2, c3;
          ldsm_x4(kh_s + k_off + (uint32_t)(nt2 * 16 * LDK * 2 + ks * 32), b0, b1, b2, b3);
          ldsm_x4(kl_s + k_off + (uint32_t)(nt2 * 16 * LDK * 2 + ks * 32), c0, c1, c2, c3);
          mma_bf16_16816(sc[2 * nt2], h0, h1, h2, h3, b0, b1);
          mma_bf16_16816(sc[2 * nt2 + 1], h0, h1, h2, h3, b2, b3);
          mma_bf16_16816(sc[2 * nt2], l0, l1, l2, l3, b0, b1);
          mma_bf16_16816(sc[2 * nt2 + 1], l0, l1, l2, l3, b2, b3);
          mma_bf16_16816(sc[2 * nt2], h0, h1, h2, h3, c0, c1);
          mma_bf16_16816(sc[2 * nt2 + 1], h0, h1, h2, h3, c2, c3);
        }
#pragma unroll
        for (int nd = 0; nd < NV / 2; ++nd) {
          uint32_t b0, b1, b2, b3, c0, c1, c2, c3;
          ldsm_x4_t(sh_s + b_off + (uint32_t)(ks * 16 * LDV * 2 + nd * 32), b0, b1, b2, b3);
          ldsm_x4_t(sl_s + b_off + (uint32_t)(ks * 16 * LDV * 2 + nd * 32), c0, c1, c2, c3);
          mma_bf16_16816(o[2 * nd], h0, h1, h2, h3, b0, b1);
          mma_bf16_16816(o[2 * nd + 1], h0, h1, h2, h3, b2, b3);
          mma_bf16_16816(o[2 * nd], l0, l1, l2, l3, b0, b1);
          mma_bf16_16816(o[2 * nd + 1], l0, l1, l2, l3, b2, b3);
          mma_bf16_16816(o[2 * nd], h0, h1, h2, h3, c0, c1);
          mma_bf16_16816(o[2 * nd + 1], h0, h1, h2, h3, c2, c3);
        }
      }
      const int i0 = warp * 16 + gq, i1 = i0 + 8;  // this thread's rows
      const float p0 = pw[i0 + 1], p1 = pw[i1 + 1];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        o[i][0] *= p0;
        o[i][1] *= p0;
        o[i][2] *= p1;
        o[i][3] *= p1;
      }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        if (kk > warp) break;
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int j = kk * 16 + u * 8 + 2 * q4;
          const float* x = sc[2 * kk + u];
          const float w00 = j <= i0 ? pw[i0 - j] : 0.f, w01 = j + 1 <= i0 ? pw[i0 - j - 1] : 0.f;
          const float w10 = j <= i1 ? pw[i1 - j] : 0.f, w11 = j + 1 <= i1 ? pw[i1 - j - 1] : 0.f;
          split_pair(x[0] * w00, x[1] * w01, ph[2 * u], pl[2 * u]);
          split_pair(x[2] * w10, x[3] * w11, ph[2 * u + 1], pl[2 * u + 1]);
        }
#pragma unroll
        for (int nd = 0; nd < NV / 2; ++nd) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4_t(v_s + b_off + (uint32_t)(kk * 16 * LDV * 2 + nd * 32), b0, b1, b2, b3);
          mma_bf16_16816(o[2 * nd], ph[0], ph[1], ph[2], ph[3], b0, b1);
          mma_bf16_16816(o[2 * nd + 1], ph[0], ph[1], ph[2], ph[3], b2, b3);
          mma_bf16_16816(o[2 * nd], pl[0], pl[1], pl[2], pl[3], b0, b1);
          mma_bf16_16816(o[2 * nd + 1], pl[0], pl[1], pl[2], pl[3], b2, b3);
        }
      }
      float* r = raw + (long long)(s.row0 + c * RCH) * HV + (long long)h * vdim + v0 + 2 * q4;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        if (i0 < n) *reinterpret_cast<float2*>(r + (long long)i0 * HV + i * 8) = make_float2(o[i][0], o[i][1]);
        if (i1 < n) *reinterpret_cast<float2*>(r + (long long)i1 * HV + i * 8) = make_float2(o[i][2], o[i][3]);
      }
    }
    // S <- lambda^n S + K^T V'
    const float pn = pw[n];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int nt = 0; nt < NV; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[m][nt][e] *= pn;
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      if (kk * 16 >= n) break;  // rows past the portion are zeros
      uint32_t bh[NV / 2][4], bl[NV / 2][4];
#pragma unroll
      for (int nd = 0; nd < NV / 2; ++nd) {
        ldsm_x4_t(vh_s + b_off + (uint32_t)(kk * 16 * LDV * 2 + nd * 32), bh[nd][0], bh[nd][1], bh[nd][2], bh[nd][3]);
        ldsm_x4_t(vl_s + b_off + (uint32_t)(kk * 16 * LDV * 2 + nd * 32), bl[nd][0], bl[nd][1], bl[nd][2], bl[nd][3]);
      }
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
        ldsm_x4_t(kh_s + kt_off + (uint32_t)((kk * 16 * LDK + m * 16) * 2), h0, h1, h2, h3);
        ldsm_x4_t(kl_s + kt_off + (uint32_t)((kk * 16 * LDK + m * 16) * 2), l0, l1, l2, l3);
#pragma unroll
        for (int nd = 0; nd < NV / 2; ++nd) {
          mma_bf16_16816(S[m][2 * nd], h0, h1, h2, h3, bh[nd][0], bh[nd][1]);
          mma_bf16_16816(S[m][2 * nd + 1], h0, h1, h2, h3, bh[nd][2], bh[nd][3]);
          mma_bf16_16816(S[m][2 * nd], l0, l1, l2, l3, bh[nd][0], bh[nd][1]);
          mma_bf16_16816(S[m][2 * nd + 1], l0, l1, l2, l3, bh[nd][2], bh[nd][3]);
          mma_bf16_16816(S[m][2 * nd], h0, h1, h2, h3, bl[nd][0], bl[nd][1]);
          mma_bf16_16816(S[m][2 * nd + 1], h0, h1, h2, h3, bl[nd][2], bl[nd][3]);
        }
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float* dst = st + (long long)(warp * (DT / 4) + m * 16 + gq + 8 * r) * vdim + n * 8 + 2 * q4;
        dst[0] = S[m][n][2 * r];
        dst[1] = S[m][n][2 * r + 1];
      }
}

// ------------------------------------------------------------------------------------------------
// norm and gate of the portions' outputs: CTA per token, warp per head
// ------------------------------------------------------------------------------------------------
template <typename T, int V>
__global__ void __launch_bounds__(256) retention_finish_kernel(const float* __restrict__ raw, const T* __restrict__ gate,
                                                               int ld_gate, int heads, int vdim, float eps,
                                                               const int32_t* __restrict__ seq_desc,
                                                               const int32_t* __restrict__ row_seq, int skip_single,
                                                               T* __restrict__ out) {
  const long long t = blockIdx.x;
  if (skip_single && seq_view(seq_desc, row_seq[t]).n == 1) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int h = warp; h < heads; h += 8) {
    const float* r = raw + (t * heads + h) * vdim;
    float ss = 0.f;
    for (int c = lane * V; c < vdim; c += 32 * V)
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(r[c + i], r[c + i], ss);
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)vdim + eps);
    const T* g = gate + t * ld_gate + (long long)h * vdim;
    T* o = out + (t * heads + h) * vdim;
    for (int c = lane * V; c < vdim; c += 32 * V)
#pragma unroll
      for (int i = 0; i < V; ++i) stf(o + c + i, r[c + i] * inv * siluf_(ldf(g + c + i)));
  }
}

}  // namespace b200q

using namespace b200q;

template <int DT, int VB>
static int launch_chunks(const bf16* qk, const bf16* v, int ldp, const float* decay, float* state, long long slot_stride,
                         const int32_t* seq_desc, int n_seqs, int heads, int vdim, float* raw, cudaStream_t st) {
  auto kern = retention_chunk_kernel<DT, VB>;
  constexpr int bytes = RetentionSmem<DT, VB>::BYTES;
  B200Q_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
  dim3 grid(n_seqs, heads, vdim / VB);
  kern<<<grid, 128, bytes, st>>>(qk, v, ldp, decay, state, slot_stride, seq_desc, heads, vdim, raw);
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

extern "C" {

int64_t b200q_retention_scratch_floats(int heads, int dim, int vdim) { return (int64_t)heads * (2 * dim + 2 * vdim); }

int b200q_retention(const void* proj, int ldp, int heads, int dim, int vdim, int rot_dims, const float* table,
                    const float* decay, float* state, long long slot_stride, const int32_t* seq_desc, const int32_t* row_seq,
                    int n_seqs, int max_portion, float eps, float* scratch, void* out, int T_, int dtype, void* stream) {
  B200Q_CHECK_ARG(proj && decay && state && seq_desc && row_seq && out && heads > 0 && heads <= 65535 && dim > 0 &&
                      dim <= 256 && vdim > 0 && vdim <= 4096 && n_seqs > 0 && T_ >= 0 && is_dtype(dtype) && eps >= 0.f &&
                      ldp >= 2 * heads * (dim + vdim),
                  "retention: bad argument (heads=%d dim=%d (<= 256) vdim=%d (<= 4096))", heads, dim, vdim);
  B200Q_CHECK_ARG(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim && (rot_dims == 0 || table),
                  "retention: rot_dims (%d) must be even and at most dim (%d)", rot_dims, dim);
  B200Q_CHECK_ARG(T_ <= n_seqs || scratch, "retention: portions need the scratch");
  if (T_ == 0) return B200Q_OK;
  cudaStream_t st = as_stream(stream);
  const int half = rot_dims / 2, HD = heads * dim, HV = heads * vdim;
  const float2* tab = (const float2*)table;
  // chunks on the tensor cores: bf16, whole tiles, 16-byte pieces
  const bool chunks = dtype == B200Q_DTYPE_BF16 && (dim == 64 || dim == 128) && vdim % 32 == 0 && half % 8 == 0 &&
                      ldp % 8 == 0 && slot_stride % 2 == 0 &&
                      ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(scratch)) & 15) == 0 &&
                      (reinterpret_cast<uintptr_t>(state) & 7) == 0;
  const bool portions = T_ > n_seqs, all_long = portions && max_portion > 1 && (long long)n_seqs * max_portion == T_;
  if (portions) {
    float* raw = scratch + (long long)T_ * 2 * HD;
    if (chunks) {
      bf16* qk = (bf16*)scratch;
      const long long total = (long long)T_ * 2 * heads * (dim / 8 - half / 8);
      retention_split_kernel<<<grid_for(total), 256, 0, st>>>((const bf16*)proj, ldp, heads, dim, half, tab, qk, total);
      B200Q_LAUNCH_CHECK();
      const bf16* v = (const bf16*)proj + 2 * HD;
      // wide value blocks repeat fewer score products, narrow ones fill more SMs
      const bool wide = vdim % 64 == 0 && (long long)n_seqs * heads * (vdim / 64) >= 148;
      int rc;
#define CHUNKS(DT, VB) \
  rc = launch_chunks<DT, VB>(qk, v, ldp, decay, state, slot_stride, seq_desc, n_seqs, heads, vdim, raw, st)
      if (dim == 64) {
        if (wide) CHUNKS(64, 64);
        else CHUNKS(64, 32);
      } else {
        if (wide) CHUNKS(128, 64);
        else CHUNKS(128, 32);
      }
#undef CHUNKS
      if (rc) return rc;
    } else {
      raw = scratch + (long long)T_ * (2 * HD + HV);
      DISPATCH_T(dtype, (retention_prep_kernel<T><<<T_, 256, 0, st>>>((const T*)proj, ldp, heads, dim, vdim, half, tab, scratch)));
      B200Q_LAUNCH_CHECK();
      if (int rc = b200q_decay_attn(scratch, 2 * HD + HV, 0, HD, 2 * HD, decay, nullptr, 0, nullptr, state, slot_stride, seq_desc,
                                    n_seqs, heads, dim, vdim, raw, stream))
        return rc;
    }
    const int skip = chunks ? 1 : 0;
    const size_t gate_at = (size_t)(2 * HD + HV);
    if (vdim % 4 == 0)
      DISPATCH_T(dtype, (retention_finish_kernel<T, 4><<<T_, 256, 0, st>>>(raw, (const T*)proj + gate_at, ldp, heads, vdim, eps,
                                                                          seq_desc, row_seq, skip, (T*)out)));
    else
      DISPATCH_T(dtype, (retention_finish_kernel<T, 1><<<T_, 256, 0, st>>>(raw, (const T*)proj + gate_at, ldp, heads, vdim, eps,
                                                                          seq_desc, row_seq, skip, (T*)out)));
    B200Q_LAUNCH_CHECK();
    if (!chunks || all_long) return B200Q_OK;  // the recurrence took the single tokens too, or there are none
  }
  const bool v4 = vdim % 4 == 0 && slot_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
  const int nc = v4 ? vdim / 4 : vdim, groups = nc < RET_THREADS ? RET_THREADS / nc : 1;
  const size_t smem = (size_t)(2 * dim + groups * vdim) * sizeof(float);
  dim3 grid(n_seqs, heads);
  if (v4)
    DISPATCH_T(dtype, (retention_decode_kernel<T, 4><<<grid, RET_THREADS, smem, st>>>(
                          (const T*)proj, ldp, heads, dim, vdim, half, tab, decay, state, slot_stride, seq_desc, eps, (T*)out)));
  else
    DISPATCH_T(dtype, (retention_decode_kernel<T, 1><<<grid, RET_THREADS, smem, st>>>(
                          (const T*)proj, ldp, heads, dim, vdim, half, tab, decay, state, slot_stride, seq_desc, eps, (T*)out)));
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

}  // extern "C"
