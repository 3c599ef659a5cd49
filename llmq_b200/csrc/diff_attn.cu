// diff_attn.cu — differential attention over a paged cache.  Every query head h and every key head g carry TWO maps
// (two queries, two keys of `dim` values each, laid out [map 1 | map 2]) over the same values; with a1, a2 the two
// softmax attentions of a head
//     o = a1 - lambda a2;   out_h = o / sqrt(mean(o^2) + eps) * mult * sigmoid(gate_h)
// lambda is one number of the layer, mult a constant, the mean runs over the head's vdim values.
//
// Step 1 (prep) turns the rows of the fused projection into queries and cache rows: biases, a short causal convolution
// of every channel of q, k and v (continued from the projected values a sequence left in its state slot), rotation of
// neighbouring dimensions (2i, 2i+1) by the step's table of cosines and sines.  A layer that borrows another layer's
// keys and values prepares queries only.
//
// Cache: [block][kv_heads][block_size][2*dim + vdim], one contiguous page per (block, key head), a row = [key 1 | key 2
// | value].  Where the tensor-core kernels run, the 16-byte pieces of row r are stored at piece index ^ (r & 7), so a
// page arrives by ONE bulk copy and is read by ldmatrix without bank conflicts.
//
// Step 2: a scalar kernel (fp32 models, any head size) and two tensor-core kernels for bf16 caches, one for portions of
// prompts (64 tokens of a head per CTA) and one for single decoded tokens (both maps of up to 8 heads are the 16 rows of
// one tile).  Scores, softmax state, accumulators, the combination of the maps and its norm are fp32 in all.
#include <stdlib.h>

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

// where element e of a cache row lies (mask 7: 16-byte pieces permuted by the row's place in its block; 0: as is)
__device__ __forceinline__ int row_place(int e, int r, int mask) { return e ^ ((r & mask) << 3); }

// ------------------------------------------------------------------------------------------------
// cosines and sines of a step: table[t][i] = (cos, sin)(position * freq[i]) * mag, angles and functions in fp64
// ------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) rot_table_kernel(const double* __restrict__ freq, float mag,
                                                        const int32_t* __restrict__ positions, int Tn, int half,
                                                        float2* __restrict__ table) {
  const int e = blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= Tn * half) return;
  double sn, c;
  sincos((double)positions[e / half] * freq[e % half], &sn, &c);
  table[e] = make_float2((float)c * mag, (float)sn * mag);
}

// what a prep kernel needs to know about the layer and the step
struct DiffPrep {
  const void* proj;        // [T, ldp]: columns [q | k | v | ...] (k and v only with own keys)
  const float* bias;       // indexed like a projection row, or NULL
  const float* conv;       // [taps][channels] or NULL
  float* state;            // this layer's part of slot 0: [taps - 1][channels], the last projected values, oldest first
  const float2* table;     // [T][rot_dims / 2]
  const int32_t *seq_desc, *row_seq, *slot_mapping;
  void* q;                 // [T, heads*2*dim], model dtype or fp32
  void* cache;
  long long slot_stride;
  float qmul;
  int ldp, heads, kv_heads, dim, vdim, taps, rot_dims, block_size, mask, own;
};

__device__ __forceinline__ long long cache_row(const DiffPrep& a, int slot, int g) {
  const int RW = 2 * a.dim + a.vdim;
  return ((long long)(slot / a.block_size) * a.kv_heads + g) * a.block_size * RW + (long long)(slot % a.block_size) * RW;
}

// any size: one thread per (token, channel); a turned channel convolves its partner too
template <typename T, typename TQ>
__global__ void __launch_bounds__(256) diff_prep_kernel(DiffPrep a) {
  const int NQ = a.heads * 2 * a.dim, NK = a.own ? a.kv_heads * 2 * a.dim : 0, NV = a.own ? a.kv_heads * a.vdim : 0;
  const int C = NQ + NK + NV, t = blockIdx.x, c = blockIdx.y * 256 + threadIdx.x;
  if (c >= C) return;
  const SeqView s = seq_view(a.seq_desc, a.row_seq[t]);
  const int tt = t - s.row0;
  const T* proj = (const T*)a.proj;
  const float* st = a.taps > 1 ? a.state + (long long)s.slot * a.slot_stride : nullptr;
  auto convolved = [&](int ch) -> float {
    const float b = a.bias ? a.bias[ch] : 0.f;
    if (!a.conv) return ldf(proj + (long long)t * a.ldp + ch) + b;
    float acc = 0.f;
    for (int j = 0; j < a.taps; ++j) {
      const int idx = tt - (a.taps - 1) + j;
      float u = 0.f;
      if (idx >= 0) u = ldf(proj + (long long)(s.row0 + idx) * a.ldp + ch) + b;
      else if (s.pos0 + idx >= 0) u = st[(long long)(a.taps - 1 + idx) * C + ch];
      acc = fmaf(a.conv[(long long)j * C + ch], u, acc);
    }
    return acc;
  };
  float y = convolved(c);
  const bool is_v = c >= NQ + NK;
  const int d = is_v ? 0 : (c < NQ ? c : c - NQ) % a.dim;
  if (!is_v && d < a.rot_dims) {
    const float2 cs = a.table[(long long)t * (a.rot_dims / 2) + d / 2];
    const float other = convolved(d & 1 ? c - 1 : c + 1);
    y = d & 1 ? y * cs.x + other * cs.y : y * cs.x - other * cs.y;
  }
  if (c < NQ) {
    stf((TQ*)a.q + (long long)t * NQ + c, y * a.qmul);
    return;
  }
  const int slot = a.slot_mapping[t];
  if (slot < 0) return;
  const int r = slot % a.block_size, ck = c - NQ, cv = c - NQ - NK;
  const int g = is_v ? cv / a.vdim : ck / (2 * a.dim);
  const int e = is_v ? 2 * a.dim + cv % a.vdim : ck % (2 * a.dim);
  stf((T*)a.cache + cache_row(a, slot, g) + row_place(e, r, a.mask), y);
}

// the carried values after the step: the last taps - 1 projected values (with bias), from the portion and, where it is
// shorter, from the old state (read completely before anything is written)
constexpr int DIFF_MAX_TAPS = 16;
template <typename T>
__global__ void __launch_bounds__(256) diff_prep_state_kernel(DiffPrep a, int skip_single) {
  const int C = a.heads * 2 * a.dim + (a.own ? a.kv_heads * (2 * a.dim + a.vdim) : 0);
  const int c = blockIdx.y * 256 + threadIdx.x;
  if (c >= C) return;
  const SeqView s = seq_view(a.seq_desc, blockIdx.x);
  if (s.n <= 0 || (skip_single && s.n == 1)) return;
  float* st = a.state + (long long)s.slot * a.slot_stride;
  const float b = a.bias ? a.bias[c] : 0.f;
  float keep[DIFF_MAX_TAPS];
#pragma unroll
  for (int i = 0; i < DIFF_MAX_TAPS; ++i) {
    if (i < a.taps - 1) {
      const int idx = s.n - (a.taps - 1) + i;
      float u = 0.f;
      if (idx >= 0) u = ldf((const T*)a.proj + (long long)(s.row0 + idx) * a.ldp + c) + b;
      else if (s.pos0 + idx >= 0) u = st[(long long)(a.taps - 1 + idx) * C + c];
      keep[i] = u;
    }
  }
#pragma unroll
  for (int i = 0; i < DIFF_MAX_TAPS; ++i)
    if (i < a.taps - 1) st[(long long)i * C + c] = keep[i];
}

// bf16, head sizes that are multiples of 8, up to 4 taps: a thread owns 8 neighbouring channels (whole rotated pairs)
// and walks up to 8 consecutive tokens of a sequence with the last values in registers.  A single token's thread also
// stores the carried values itself: nobody else reads them.
constexpr int PREP_TOKENS = 8;
template <int TAPS>
__global__ void __launch_bounds__(128) diff_prep_v8_kernel(DiffPrep a) {
  const int NQ = a.heads * 2 * a.dim, NK = a.own ? a.kv_heads * 2 * a.dim : 0, NV = a.own ? a.kv_heads * a.vdim : 0;
  const int C = NQ + NK + NV, c = (blockIdx.y * 128 + threadIdx.x) * 8;
  const SeqView s = seq_view(a.seq_desc, blockIdx.x);
  const int r0 = blockIdx.z * PREP_TOKENS;
  if (c >= C || r0 >= s.n) return;
  const int n = min(PREP_TOKENS, s.n - r0);
  const bf16* proj = (const bf16*)a.proj + (long long)(s.row0 + r0) * a.ldp + c;
  float bias[8], w[TAPS][8], hist[TAPS > 1 ? TAPS - 1 : 1][8];  // hist[i]: the value TAPS - 1 - i tokens back
  auto ld8 = [](const float* p, float (&v)[8]) {
    const float4 x = *reinterpret_cast<const float4*>(p), y = *reinterpret_cast<const float4*>(p + 4);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    v[4] = y.x; v[5] = y.y; v[6] = y.z; v[7] = y.w;
  };
  auto ldb8 = [](const bf16* p, float (&v)[8]) {
    const uint4 u = ld_v4(p);
    const uint32_t x[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      v[2 * i] = bf16_lo(x[i]);
      v[2 * i + 1] = bf16_hi(x[i]);
    }
  };
  if (a.bias) ld8(a.bias + c, bias);
  else
#pragma unroll
    for (int i = 0; i < 8; ++i) bias[i] = 0.f;
  if (a.conv) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) ld8(a.conv + (long long)j * C + c, w[j]);
  }
  float* st = TAPS > 1 ? a.state + (long long)s.slot * a.slot_stride + c : nullptr;
#pragma unroll
  for (int i = 0; i < TAPS - 1; ++i) {
    const int idx = r0 - (TAPS - 1) + i;  // relative to the portion's first token
    if (idx >= 0) {
      ldb8(proj + (long long)(idx - r0) * a.ldp, hist[i]);
#pragma unroll
      for (int k = 0; k < 8; ++k) hist[i][k] += bias[k];
    } else if (s.pos0 + idx >= 0) {
      ld8(st + (long long)(TAPS - 1 + idx) * C, hist[i]);
    } else {
#pragma unroll
      for (int k = 0; k < 8; ++k) hist[i][k] = 0.f;
    }
  }
  const bool is_q = c < NQ, is_v = c >= NQ + NK;
  const int d = is_v ? 0 : (is_q ? c : c - NQ) % a.dim, half = a.rot_dims / 2;
  const int pairs = is_v ? 0 : max(0, min(4, (a.rot_dims - d) / 2));  // rotated pairs among the 8 channels
  const int cv = c - NQ - NK, ck = c - NQ;
  const int g = is_v ? cv / a.vdim : ck / (2 * a.dim), e = is_v ? 2 * a.dim + cv % a.vdim : ck % (2 * a.dim);
  uint4 next = ld_v4(proj);
  for (int i = 0; i < n; ++i) {
    const long long t = s.row0 + r0 + i;
    const uint32_t raw[4] = {next.x, next.y, next.z, next.w};
    if (i + 1 < n) next = ld_v4(proj + (long long)(i + 1) * a.ldp);  // in flight while this token is worked on
    float u[8], y[8];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      u[2 * k] = bf16_lo(raw[k]);
      u[2 * k + 1] = bf16_hi(raw[k]);
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      u[k] += bias[k];
      if (a.conv) {
        float acc = 0.f;
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) acc = fmaf(w[j][k], hist[j][k], acc);
        y[k] = fmaf(w[TAPS - 1][k], u[k], acc);
      } else {
        y[k] = u[k];
      }
    }
#pragma unroll
    for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
      for (int k = 0; k < 8; ++k) hist[j][k] = hist[j + 1][k];
    if (TAPS > 1) {
#pragma unroll
      for (int k = 0; k < 8; ++k) hist[TAPS > 1 ? TAPS - 2 : 0][k] = u[k];
    }
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (k < pairs) {
        const float2 cs = a.table[t * half + d / 2 + k];
        const float p = y[2 * k], q = y[2 * k + 1];
        y[2 * k] = p * cs.x - q * cs.y;
        y[2 * k + 1] = q * cs.x + p * cs.y;
      }
    const float mul = is_q ? a.qmul : 1.f;
    const uint4 o = make_uint4(pack_bf16x2(y[0] * mul, y[1] * mul), pack_bf16x2(y[2] * mul, y[3] * mul),
                               pack_bf16x2(y[4] * mul, y[5] * mul), pack_bf16x2(y[6] * mul, y[7] * mul));
    if (is_q) {
      st_v4((bf16*)a.q + t * NQ + c, o);
    } else {
      const int slot = a.slot_mapping[t];
      if (slot >= 0) st_v4((bf16*)a.cache + cache_row(a, slot, g) + row_place(e, slot % a.block_size, a.mask), o);
    }
  }
  if (TAPS > 1 && s.n == 1) {
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) {
      *reinterpret_cast<float4*>(st + (long long)i * C) = make_float4(hist[i][0], hist[i][1], hist[i][2], hist[i][3]);
      *reinterpret_cast<float4*>(st + (long long)i * C + 4) = make_float4(hist[i][4], hist[i][5], hist[i][6], hist[i][7]);
    }
  }
}

// what the attention kernels need
struct DiffAttn {
  const void* q;  // [T, heads, 2, dim], scale folded in (scalar form: fp32; tensor-core form: bf16, scale * log2 e)
  const void* cache;
  const int32_t *block_table, *seq_desc, *row_seq, *positions;
  const float* lambda;
  const void* gate;  // one number per head, rows of stride ld_gate, or NULL
  void* out;         // [T, ld_out]: head h's values at h*vdim
  int* failed;       // set when a bounded wait runs out
  float mult, eps;
  int bt_stride, heads, kv_heads, dim, vdim, block_size, ld_gate, ld_out, mask;
};

// ------------------------------------------------------------------------------------------------
// scalar form: one CTA per (token, key head, group of 4 query heads); warp = (head, map).  Tiles of 32 cached rows are
// staged in shared memory once for all eight maps (lane = key for the scores, lane = value channels for the weighted
// sum).  Tiles start at key 0, so a token's result does not depend on what else the step holds.
// ------------------------------------------------------------------------------------------------
template <typename T, int ACC>
__global__ void __launch_bounds__(256) diff_attn_kernel(DiffAttn a) {
  extern __shared__ float sm[];
  const int dim = a.dim, vdim = a.vdim, RW = 2 * dim + vdim, KS = 2 * dim + 1, VS = vdim + 1;
  float* qsm = sm;                 // [8][dim]
  float* ksm = sm + 8 * dim;       // [32][2*dim + 1]
  float* vsm = ksm + 32 * KS;      // [32][vdim + 1]
  const int t = blockIdx.x, g = blockIdx.y, rep = a.heads / a.kv_heads;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, map = warp & 1;
  const int hg = blockIdx.z * 4 + (warp >> 1);
  const bool live = hg < rep;
  const int h = g * rep + hg;
  const int p = a.positions[t];
  const int32_t* bt = a.block_table + (long long)a.row_seq[t] * a.bt_stride;
  const float* q = (const float*)a.q;
  for (int e = threadIdx.x; e < 8 * dim; e += blockDim.x) {
    const int hh = blockIdx.z * 4 + e / (2 * dim);
    qsm[e] = hh < rep ? q[((long long)t * a.heads + g * rep + hh) * 2 * dim + e % (2 * dim)] : 0.f;
  }
  float m = -INFINITY, l = 0.f;
  float acc[ACC];
#pragma unroll
  for (int i = 0; i < ACC; ++i) acc[i] = 0.f;
  const float* qh = qsm + warp * dim;
  for (int j0 = 0; j0 <= p; j0 += 32) {
    const int n = min(32, p + 1 - j0);
    __syncthreads();
    for (int e = threadIdx.x; e < n * RW; e += blockDim.x) {
      const int j = e / RW, d = e % RW, pos = j0 + j, r = pos % a.block_size;
      const T* row = (const T*)a.cache +
                     ((long long)bt[pos / a.block_size] * a.kv_heads + g) * a.block_size * RW + (long long)r * RW;
      const float v = ldf(row + row_place(d, r, a.mask));
      if (d < 2 * dim) ksm[j * KS + d] = v;
      else vsm[j * VS + d - 2 * dim] = v;
    }
    __syncthreads();
    if (!live) continue;
    float s = -INFINITY;
    if (lane < n) {
      const float* kr = ksm + lane * KS + map * dim;
      float dot = 0.f;
      for (int d = 0; d < dim; ++d) dot = fmaf(qh[d], kr[d], dot);
      s = dot;
    }
    const float m_new = fmaxf(m, warp_max(s));  // the tile holds at least one visible key: finite
    const float corr = expf(m - m_new);
    const float pl = lane < n ? expf(s - m_new) : 0.f;
    l = l * corr + warp_sum(pl);
#pragma unroll
    for (int i = 0; i < ACC; ++i) acc[i] *= corr;
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, pl, j);
      const float* vr = vsm + j * VS;
#pragma unroll
      for (int i = 0; i < ACC; ++i) {
        const int d = lane + 32 * i;
        if (d < vdim) acc[i] = fmaf(pj, vr[d], acc[i]);
      }
    }
    m = m_new;
  }
  // the second map hands its output to the first map's warp through the key tile's space
  __syncthreads();
  float* osm = ksm;  // [4][vdim]: 4*vdim <= 32*(2*dim + 1 + vdim + 1)
  if (live && map == 1) {
#pragma unroll
    for (int i = 0; i < ACC; ++i) {
      const int d = lane + 32 * i;
      if (d < vdim) osm[(warp >> 1) * vdim + d] = acc[i] / l;
    }
  }
  __syncthreads();
  if (!live || map == 1) return;
  const float lam = a.lambda[0];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < ACC; ++i) {
    const int d = lane + 32 * i;
    if (d < vdim) {
      acc[i] = acc[i] / l - lam * osm[(warp >> 1) * vdim + d];
      ss = fmaf(acc[i], acc[i], ss);
    }
  }
  const float gv = a.gate ? sigmoidf_(ldf((const T*)a.gate + (long long)t * a.ld_gate + h)) : 1.f;
  const float f = a.mult * gv / sqrtf(warp_sum(ss) / (float)vdim + a.eps);
  T* o = (T*)a.out + (long long)t * a.ld_out + h * vdim;
#pragma unroll
  for (int i = 0; i < ACC; ++i) {
    const int d = lane + 32 * i;
    if (d < vdim) stf(o + d, acc[i] * f);
  }
}

constexpr float DATT_NEG = -1e30f;  // finite floor of the running maximum: exp2(masked - floor) = 0, never NaN
constexpr int DATT_PAGE = 16;       // cached rows of a page (= block size)

// ------------------------------------------------------------------------------------------------
// portions of prompts: one CTA of 4 warps per (sequence, head, 64 consecutive tokens); warp w owns 16 of them.  Tiles of
// 64 cached rows (4 pages, each one bulk copy) pass through a ring of STG stages; both maps of the head use the same
// values, so a value fragment is read from shared memory once for two products.  Weights are rounded to bf16 before they
// are summed, as the value product sees them.  Heavy tiles (late tokens) are launched first.
// ------------------------------------------------------------------------------------------------
template <int DM, int VM, int STG>
__global__ void __launch_bounds__(128, DM <= 64 ? 2 : 1) diff_attn_tile_kernel(DiffAttn a, int skip_single) {
  extern __shared__ __align__(128) uint8_t smraw[];
  __shared__ __align__(8) uint64_t full[STG];
  const int dim = a.dim, vdim = a.vdim, RW = 2 * dim + vdim, RWB = RW * 2, LDQ = (2 * dim + 63) & ~63;
  uint8_t* ring = smraw;                                                // [STG][64][RW] bf16
  bf16* qsm = reinterpret_cast<bf16*>(smraw + (size_t)STG * 64 * RWB);  // [64][LDQ], pieces permuted like the cache's
  const SeqView sq = seq_view(a.seq_desc, blockIdx.x);
  const int r0 = (gridDim.z - 1 - blockIdx.z) * 64;
  if (r0 >= sq.n || (skip_single && sq.n == 1)) return;  // single tokens: the decode kernel's
  const int nrows = min(64, sq.n - r0), h = blockIdx.y, g = h / (a.heads / a.kv_heads);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, q4 = lane & 3;
  const int p_first = sq.pos0 + r0, p_last = p_first + nrows - 1;
  const int32_t* bt = a.block_table + (long long)blockIdx.x * a.bt_stride;
  const int ntiles = p_last / 64 + 1;
  if (tid == 0) {
#pragma unroll
    for (int i = 0; i < STG; ++i) mbar_init(full + i, 1);
    mbar_fence_init();
  }
  __syncthreads();
  auto issue = [&](int c) {  // by thread 0: the valid rows of tile c, page by page
    const int stage = c % STG, valid = min(64, p_last + 1 - c * 64);
    mbar_expect_tx(full + stage, (uint32_t)(valid * RWB));
    for (int pg = 0; pg * DATT_PAGE < valid; ++pg) {
      const long long page = ((long long)bt[c * 4 + pg] * a.kv_heads + g) * DATT_PAGE * RW;
      tma_bulk_g2s(ring + (size_t)(stage * 64 + pg * DATT_PAGE) * RWB, (const bf16*)a.cache + page,
                   (uint32_t)(min(DATT_PAGE, valid - pg * DATT_PAGE) * RWB), full + stage);
    }
  };
  if (tid == 0)
    for (int c = 0; c < STG - 1 && c < ntiles; ++c) issue(c);
  // the queries of the tile; rows past the portion are zeros
  {
    const int per = 2 * dim / 8;
    for (int e = tid; e < 64 * per; e += 128) {
      const int r = e / per, ck = e % per;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < nrows) v = ld_v4((const bf16*)a.q + ((long long)(sq.row0 + r0 + r) * a.heads + h) * 2 * dim + ck * 8);
      st_v4(qsm + r * LDQ + ((ck ^ (r & 7)) * 8), v);
    }
  }
  const uint32_t q_s = smem_u32(qsm + (warp * 16 + (lane & 15)) * LDQ);
  const int krow = (lane & 7) + 8 * (lane >> 4), kck = (lane >> 3) & 1;  // key fragments: row of 16, piece of 2
  const int vrow = ((lane >> 3) & 1) * 8 + (lane & 7), vck = lane >> 4, swz = lane & 7;
  int p_row[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int i = warp * 16 + gq + 8 * r;
    p_row[r] = i < nrows ? p_first + i : -1;  // a dead row sees no key
  }
  const int w_first = p_first + warp * 16, w_last = min(w_first + 15, p_last);
  const bool warp_live = warp * 16 < nrows;
  float m_[2][2], l_[2][2], o[2][VM / 8][4];
#pragma unroll
  for (int mp = 0; mp < 2; ++mp) {
    m_[mp][0] = m_[mp][1] = DATT_NEG;
    l_[mp][0] = l_[mp][1] = 0.f;
#pragma unroll
    for (int i = 0; i < VM / 8; ++i) o[mp][i][0] = o[mp][i][1] = o[mp][i][2] = o[mp][i][3] = 0.f;
  }
  for (int c = 0; c < ntiles; ++c) {
    const int stage = c % STG, j0 = c * 64;
    bool ok = mbar_wait_limited(full + stage, (uint32_t)(c / STG) & 1u);
    if (c == ntiles - 1) {  // rows past the last token: their weights are zeros, their values must not be NaNs
      const int valid = p_last + 1 - j0, per = vdim / 8;
      for (int e = tid; e < (64 - valid) * per; e += 128) {
        const int r = valid + e / per, ck = 2 * dim / 8 + e % per;
        st_v4(ring + (size_t)(stage * 64 + r) * RWB + ((ck ^ (r & 7)) << 4), make_uint4(0, 0, 0, 0));
      }
    }
    ok = __syncthreads_and(ok);  // tile c is whole for everyone, tile c - 1 is done with
    if (!ok) {  // give up: let the copies already on their way land first
      if (tid == 0) {
        for (int i = c + 1; i < c + STG - 1 && i < ntiles; ++i) mbar_wait_limited(full + i % STG, (uint32_t)(i / STG) & 1u);
        *(volatile int*)a.failed = 1;
      }
      return;
    }
    if (tid == 0 && c + STG - 1 < ntiles) issue(c + STG - 1);
    if (!warp_live || j0 > w_last) continue;
    const uint32_t tb = smem_u32(ring + (size_t)stage * 64 * RWB);
    uint32_t pk[2][16];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
      float s[8][4];
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
      const int ck0 = mp * (dim / 8);
#pragma unroll
      for (int ks = 0; ks < DM / 16; ++ks) {
        if (ks * 16 >= dim) break;
        uint32_t a0, a1, a2, a3;
        ldsm_x4(q_s + (uint32_t)(((ck0 + ks * 2 + (lane >> 4)) ^ swz) << 4), a0, a1, a2, a3);
        const uint32_t kp = tb + (uint32_t)(krow * RWB) + (uint32_t)(((ck0 + ks * 2 + kck) ^ swz) << 4);
#pragma unroll
        for (int nt2 = 0; nt2 < 4; ++nt2) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4(kp + (uint32_t)(nt2 * 16 * RWB), b0, b1, b2, b3);
          mma_bf16_16816(s[2 * nt2], a0, a1, a2, a3, b0, b1);
          mma_bf16_16816(s[2 * nt2 + 1], a0, a1, a2, a3, b2, b3);
        }
      }
      if (j0 + 63 > w_first || nrows < 64) {
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (j0 + nt * 8 + 2 * q4 + (e & 1) > p_row[e >> 1]) s[nt][e] = -INFINITY;
      }
      float corr[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float mx = DATT_NEG;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) mx = fmaxf(mx, fmaxf(s[nt][2 * r], s[nt][2 * r + 1]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float mn = fmaxf(m_[mp][r], mx);
        corr[r] = exp2f(m_[mp][r] - mn);
        m_[mp][r] = mn;
        float ps = 0.f;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
          const float e0 = exp2f(s[nt][2 * r] - mn), e1 = exp2f(s[nt][2 * r + 1] - mn);  // masked: exp2(-inf) = 0
          const uint32_t v = pack_bf16x2(e0, e1);
          ps += bf16_lo(v) + bf16_hi(v);
          pk[mp][(nt >> 1) * 4 + (nt & 1) * 2 + r] = v;
        }
        l_[mp][r] = l_[mp][r] * corr[r] + ps;
      }
      if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
        for (int i = 0; i < VM / 8; ++i) {
          o[mp][i][0] *= corr[0];
          o[mp][i][1] *= corr[0];
          o[mp][i][2] *= corr[1];
          o[mp][i][3] *= corr[1];
        }
      }
    }
    const int vc0 = 2 * dim / 8;
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      const uint32_t vp = tb + (uint32_t)((kk * 16 + vrow) * RWB);
#pragma unroll
      for (int nd = 0; nd < VM / 16; ++nd) {
        if (nd * 16 >= vdim) break;
        uint32_t b0, b1, b2, b3;
        ldsm_x4_t(vp + (uint32_t)(((vc0 + nd * 2 + vck) ^ swz) << 4), b0, b1, b2, b3);
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
          mma_bf16_16816(o[mp][2 * nd], pk[mp][4 * kk], pk[mp][4 * kk + 1], pk[mp][4 * kk + 2], pk[mp][4 * kk + 3], b0, b1);
          mma_bf16_16816(o[mp][2 * nd + 1], pk[mp][4 * kk], pk[mp][4 * kk + 1], pk[mp][4 * kk + 2], pk[mp][4 * kk + 3], b2,
                         b3);
        }
      }
    }
  }
  if (!warp_live) return;
  const float lam = a.lambda[0];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float inv[2];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
      float l = l_[mp][r];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      inv[mp] = 1.f / l;
    }
    inv[1] *= lam;
    float ss = 0.f;
#pragma unroll
    for (int nt = 0; nt < VM / 8; ++nt) {
      if (nt * 8 >= vdim) break;
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const float v = o[0][nt][2 * r + k] * inv[0] - o[1][nt][2 * r + k] * inv[1];
        o[0][nt][2 * r + k] = v;
        ss = fmaf(v, v, ss);
      }
    }
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    if (p_row[r] < 0) continue;
    const long long t = sq.row0 + (p_row[r] - sq.pos0);
    const float gv = a.gate ? sigmoidf_(__bfloat162float(((const bf16*)a.gate)[t * a.ld_gate + h])) : 1.f;
    const float f = a.mult * gv / sqrtf(ss / (float)vdim + a.eps);
    bf16* orow = (bf16*)a.out + t * a.ld_out + h * vdim;
#pragma unroll
    for (int nt = 0; nt < VM / 8; ++nt) {
      if (nt * 8 >= vdim) break;
      *reinterpret_cast<uint32_t*>(orow + nt * 8 + 2 * q4) = pack_bf16x2(o[0][nt][2 * r] * f, o[0][nt][2 * r + 1] * f);
    }
  }
}

// ------------------------------------------------------------------------------------------------
// single decoded tokens: one CTA of 4 warps per (sequence, key head, 8 query heads).  Row r < 8 of the tile is map 1 of
// head r, row 8 + r its map 2; the query rows are [q1 | 0] and [0 | q2], so one product over the 2*dim key columns gives
// both maps' scores and one pass over a page serves all of them.  Warp w takes the pages w, w + 4, ... through its own
// ring of bulk copies (no CTA barrier inside the loop) and keeps its own softmax state; the four states are merged in a
// fixed order at the end, where the maps are combined and normed.
// ------------------------------------------------------------------------------------------------
constexpr int DDEC_WARPS = 4;
template <int DM, int VM, int STG>
__global__ void __launch_bounds__(128) diff_attn_decode_kernel(DiffAttn a) {
  extern __shared__ __align__(128) uint8_t smraw[];
  __shared__ __align__(8) uint64_t full[DDEC_WARPS][STG];
  const int dim = a.dim, vdim = a.vdim, RW = 2 * dim + vdim, RWB = RW * 2, LDQ = 2 * dim + 8, MS = vdim + 2;
  const SeqView sq = seq_view(a.seq_desc, blockIdx.x);
  if (sq.n != 1) return;  // portions of prompts take the tile kernel
  const int rep = a.heads / a.kv_heads, parts = (rep + 7) / 8, g = blockIdx.y / parts, h0 = (blockIdx.y % parts) * 8;
  const int nh = min(8, rep - h0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, q4 = lane & 3;
  const int p = sq.pos0, npages = p / DATT_PAGE + 1;
  const long long t = sq.row0;
  const int32_t* bt = a.block_table + (long long)blockIdx.x * a.bt_stride;
  const size_t page_bytes = (size_t)DATT_PAGE * RWB;
  uint8_t* ring = smraw + (size_t)warp * STG * page_bytes;                                 // [4 warps][STG][16][RW] bf16
  bf16* qsm = reinterpret_cast<bf16*>(smraw + (size_t)DDEC_WARPS * STG * page_bytes);      // [16][LDQ]
  uint64_t* bars = full[warp];
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < STG; ++i) mbar_init(bars + i, 1);
    mbar_fence_init();
  }
  __syncwarp();
  // lane i holds the block of this warp's page number base + i
  int base = 0;
  auto blocks_from = [&](int b) -> int {
    const int c = warp + DDEC_WARPS * (b + lane);
    return c < npages ? bt[c] : 0;
  };
  int blk = blocks_from(0);
  auto issue = [&](int it) {  // whole warp: page warp + 4*it into stage it % STG
    const int c = warp + DDEC_WARPS * it;
    if (it - base >= 32) {
      base = it;
      blk = blocks_from(base);
    }
    const int b = __shfl_sync(0xffffffffu, blk, it - base);
    if (lane == 0) {
      const uint32_t bytes = (uint32_t)(min(DATT_PAGE, p + 1 - c * DATT_PAGE) * RWB);
      mbar_expect_tx(bars + it % STG, bytes);
      tma_bulk_g2s(ring + (size_t)(it % STG) * page_bytes,
                   (const bf16*)a.cache + ((long long)b * a.kv_heads + g) * DATT_PAGE * RW, bytes, bars + it % STG);
    }
  };
  const int n_it = warp < npages ? (npages - warp + DDEC_WARPS - 1) / DDEC_WARPS : 0;
  for (int it = 0; it < STG && it < n_it; ++it) issue(it);
  {
    const int per = 2 * dim / 8;  // 16-byte pieces of a row; the other map's half is zeros
    for (int e = tid; e < 16 * per; e += 128) {
      const int r = e / per, ck = e % per, map = r >> 3, hh = r & 7;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (hh < nh && ck / (dim / 8) == map)
        v = ld_v4((const bf16*)a.q + (t * a.heads + g * rep + h0 + hh) * 2 * dim + ck * 8);
      st_v4(qsm + r * LDQ + ck * 8, v);
    }
  }
  __syncthreads();
  const uint32_t q_s = smem_u32(qsm) + (uint32_t)(((lane & 15) * LDQ + (lane >> 4) * 8) * 2);
  uint32_t qa[2 * DM / 16][4];
#pragma unroll
  for (int ks = 0; ks < 2 * DM / 16; ++ks)
    if (ks * 16 < 2 * dim) ldsm_x4(q_s + (uint32_t)(ks * 32), qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3]);
  const int krow = (lane & 7) + 8 * (lane >> 4), kck = (lane >> 3) & 1;
  const int vrow = ((lane >> 3) & 1) * 8 + (lane & 7), vck = lane >> 4, swz = lane & 7;
  const bool row_on = gq < nh;  // rows gq (map 1) and gq + 8 (map 2) are the same head's
  float m_[2] = {DATT_NEG, DATT_NEG}, l_[2] = {0.f, 0.f};
  float o[VM / 8][4];
#pragma unroll
  for (int i = 0; i < VM / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  bool ok = true;
  for (int it = 0; it < n_it; ++it) {
    const int stage = it % STG, j0 = (warp + DDEC_WARPS * it) * DATT_PAGE;
    ok = mbar_wait_limited(bars + stage, (uint32_t)(it / STG) & 1u);
    if (!__all_sync(0xffffffffu, ok)) {  // give up: let the copies already on their way land first
      for (int i = it + 1; i < it + STG && i < n_it; ++i) mbar_wait_limited(bars + i % STG, (uint32_t)(i / STG) & 1u);
      ok = false;
      break;
    }
    uint8_t* page = ring + (size_t)stage * page_bytes;
    if (j0 + DATT_PAGE > p + 1) {  // rows past the token: their weights are zeros, their values must not be NaNs
      const int valid = p + 1 - j0, per = vdim / 8;
      for (int e = lane; e < (DATT_PAGE - valid) * per; e += 32) {
        const int r = valid + e / per, ck = 2 * dim / 8 + e % per;
        st_v4(page + (size_t)r * RWB + ((ck ^ (r & 7)) << 4), make_uint4(0, 0, 0, 0));
      }
      __syncwarp();
    }
    const uint32_t tb = smem_u32(page);
    float s[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < 2 * DM / 16; ++ks) {
      if (ks * 16 >= 2 * dim) break;
      uint32_t b0, b1, b2, b3;
      ldsm_x4(tb + (uint32_t)(krow * RWB) + (uint32_t)(((ks * 2 + kck) ^ swz) << 4), b0, b1, b2, b3);
      mma_bf16_16816(s[0], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], b0, b1);
      mma_bf16_16816(s[1], qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3], b2, b3);
    }
    uint32_t pk[4];
    float corr[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float mx = DATT_NEG;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          if (!row_on || j0 + nt * 8 + 2 * q4 + k > p) s[nt][2 * r + k] = -INFINITY;
          mx = fmaxf(mx, s[nt][2 * r + k]);
        }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float mn = fmaxf(m_[r], mx);
      corr[r] = exp2f(m_[r] - mn);
      m_[r] = mn;
      float ps = 0.f;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        const uint32_t v = pack_bf16x2(exp2f(s[nt][2 * r] - mn), exp2f(s[nt][2 * r + 1] - mn));
        ps += bf16_lo(v) + bf16_hi(v);
        pk[nt * 2 + r] = v;
      }
      l_[r] = l_[r] * corr[r] + ps;
    }
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int i = 0; i < VM / 8; ++i) {
        o[i][0] *= corr[0];
        o[i][1] *= corr[0];
        o[i][2] *= corr[1];
        o[i][3] *= corr[1];
      }
    }
    const uint32_t vp = tb + (uint32_t)(vrow * RWB);
#pragma unroll
    for (int nd = 0; nd < VM / 16; ++nd) {
      if (nd * 16 >= vdim) break;
      uint32_t b0, b1, b2, b3;
      ldsm_x4_t(vp + (uint32_t)(((2 * dim / 8 + nd * 2 + vck) ^ swz) << 4), b0, b1, b2, b3);
      mma_bf16_16816(o[2 * nd], pk[0], pk[1], pk[2], pk[3], b0, b1);
      mma_bf16_16816(o[2 * nd + 1], pk[0], pk[1], pk[2], pk[3], b2, b3);
    }
    __syncwarp();  // every lane is done with the stage
    if (it + STG < n_it) issue(it + STG);
  }
  // ---- merge the four warps' states: [warp][row][vdim + 2] = (o..., m, l); a warp without pages holds (0, floor, 0) ----
  ok = __syncthreads_and(ok);  // every warp is done with its ring: it becomes the merge area
  if (!ok) {
    if (tid == 0) *(volatile int*)a.failed = 1;
    return;
  }
  float* mrg = reinterpret_cast<float*>(smraw);
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_[r] += __shfl_xor_sync(0xffffffffu, l_[r], 1);
    l_[r] += __shfl_xor_sync(0xffffffffu, l_[r], 2);
    float* dst = mrg + (size_t)(warp * 16 + gq + 8 * r) * MS;
#pragma unroll
    for (int nt = 0; nt < VM / 8; ++nt) {
      if (nt * 8 >= vdim) break;
      dst[nt * 8 + 2 * q4] = o[nt][2 * r];
      dst[nt * 8 + 2 * q4 + 1] = o[nt][2 * r + 1];
    }
    if (q4 == 0) {
      dst[vdim] = m_[r];
      dst[vdim + 1] = l_[r];
    }
  }
  __syncthreads();
  const float lam = a.lambda[0];
  for (int hh = warp; hh < nh; hh += DDEC_WARPS) {  // one warp per head
    float f[2][DDEC_WARPS], inv[2];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
      float mx = DATT_NEG, den = 0.f;
#pragma unroll
      for (int w = 0; w < DDEC_WARPS; ++w) mx = fmaxf(mx, mrg[(size_t)(w * 16 + hh + 8 * mp) * MS + vdim]);
#pragma unroll
      for (int w = 0; w < DDEC_WARPS; ++w) {
        f[mp][w] = exp2f(mrg[(size_t)(w * 16 + hh + 8 * mp) * MS + vdim] - mx);
        den = fmaf(mrg[(size_t)(w * 16 + hh + 8 * mp) * MS + vdim + 1], f[mp][w], den);
      }
      inv[mp] = 1.f / den;
    }
    float v[VM / 32], ss = 0.f;
#pragma unroll
    for (int i = 0; i < VM / 32; ++i) {
      const int d = lane + 32 * i;
      v[i] = 0.f;
      if (d < vdim) {
        float num[2] = {0.f, 0.f};
#pragma unroll
        for (int mp = 0; mp < 2; ++mp)
#pragma unroll
          for (int w = 0; w < DDEC_WARPS; ++w) num[mp] = fmaf(mrg[(size_t)(w * 16 + hh + 8 * mp) * MS + d], f[mp][w], num[mp]);
        v[i] = num[0] * inv[0] - lam * (num[1] * inv[1]);
        ss = fmaf(v[i], v[i], ss);
      }
    }
    const int h = g * rep + h0 + hh;
    const float gv = a.gate ? sigmoidf_(__bfloat162float(((const bf16*)a.gate)[t * a.ld_gate + h])) : 1.f;
    const float fac = a.mult * gv / sqrtf(warp_sum(ss) / (float)vdim + a.eps);
#pragma unroll
    for (int i = 0; i < VM / 32; ++i) {
      const int d = lane + 32 * i;
      if (d < vdim) ((bf16*)a.out)[t * a.ld_out + h * vdim + d] = __float2bfloat16_rn(v[i] * fac);
    }
  }
}

// one flag in mapped host memory for the process: a kernel whose wait ran out sets it, the host reads it without a copy
int* wait_flag(int** dev) {
  static int *host = nullptr, *device = nullptr;
  if (!host) {
    if (cudaHostAlloc((void**)&host, 64, cudaHostAllocMapped) != cudaSuccess) return nullptr;
    *host = 0;
    if (cudaHostGetDevicePointer((void**)&device, host, 0) != cudaSuccess) return nullptr;
  }
  if (dev) *dev = device;
  return host;
}

}  // namespace b200q

using namespace b200q;

// most tokens of a portion: what the caller says, or what a step of T tokens leaves for one of n_seqs sequences
static int longest_portion(int max_portion, int n_seqs, int T) {
  const int bound = T - n_seqs + 1;
  return max_portion > 0 && max_portion < bound ? max_portion : bound;
}

static bool diff_attn_mma_mode() {  // B200Q_DIFF_ATTN_MMA=0: the scalar kernels everywhere
  static const bool on = [] {
    const char* v = getenv("B200Q_DIFF_ATTN_MMA");
    return !v || atoi(v) != 0;
  }();
  return on;
}

template <int DM, int VM>
static int launch_diff_mma(const DiffAttn& a, int n_seqs, int longest, int T, cudaStream_t st) {
  constexpr int STG = DM <= 64 ? 3 : 2, DSTG = DM <= 64 ? 3 : 2;
  const int RW = 2 * a.dim + a.vdim, rep = a.heads / a.kv_heads, parts = (rep + 7) / 8;
  if (T > n_seqs) {  // portions of prompts
    dim3 grid(n_seqs, a.heads, (longest + 63) / 64);
    B200Q_CHECK_ARG(grid.y <= 65535 && grid.z <= 65535, "diff_attn: step too large (%d tokens)", T);
    const size_t smem = (size_t)STG * 64 * RW * 2 + (size_t)64 * ((2 * a.dim + 63) & ~63) * 2;
    auto kern = diff_attn_tile_kernel<DM, VM, STG>;
    if (smem > 48 * 1024) B200Q_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    kern<<<grid, 128, smem, st>>>(a, 1);
    B200Q_LAUNCH_CHECK();
    if ((long long)n_seqs * longest == T) return B200Q_OK;  // every portion is as long: no single tokens
  }
  dim3 grid(n_seqs, a.kv_heads * parts);
  B200Q_CHECK_ARG(grid.y <= 65535, "diff_attn: too many heads");
  const size_t smem = std::max((size_t)DDEC_WARPS * DSTG * DATT_PAGE * RW * 2 + (size_t)16 * (2 * a.dim + 8) * 2,
                               (size_t)DDEC_WARPS * 16 * (a.vdim + 2) * 4);
  auto kern = diff_attn_decode_kernel<DM, VM, DSTG>;
  if (smem > 48 * 1024) B200Q_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  kern<<<grid, 128, smem, st>>>(a);
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

extern "C" {

int b200q_diff_attn_tiled(int dim, int vdim, int block_size, int dtype) {
  return dtype == B200Q_DTYPE_BF16 && block_size == DATT_PAGE && dim > 0 && dim % 16 == 0 && dim <= 128 && vdim > 0 &&
                 vdim % 16 == 0 && vdim <= 128 && (2 * dim + vdim) % 64 == 0 && diff_attn_mma_mode()
             ? 1
             : 0;
}

int b200q_wait_failures(void) {
  int* f = wait_flag(nullptr);
  return f ? *(volatile int*)f : 0;
}

int b200q_rot_table(const double* freq, float mag, const int32_t* positions, int T_, int half, float* table, void* stream) {
  B200Q_CHECK_ARG(freq && positions && table && T_ >= 0 && half > 0 && (long long)T_ * half < (1ll << 31),
                  "rot_table: bad argument (T=%d half=%d)", T_, half);
  if (T_ == 0) return B200Q_OK;
  rot_table_kernel<<<(T_ * half + 255) / 256, 256, 0, as_stream(stream)>>>(freq, mag, positions, T_, half, (float2*)table);
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

int b200q_diff_attn_prep(const void* proj, int ldp, const float* bias, const float* conv, int taps, float* state,
                         long long slot_stride, int own, int heads, int kv_heads, int dim, int vdim, int rot_dims,
                         const float* table, float scale, const int32_t* seq_desc, const int32_t* row_seq, int n_seqs,
                         int max_portion, const int32_t* slot_mapping, int block_size, void* q, void* cache, int T_, int dtype,
                         void* stream) {
  B200Q_CHECK_ARG(proj && q && seq_desc && row_seq && n_seqs > 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 &&
                      dim > 0 && vdim > 0 && block_size > 0 && T_ >= 0 && is_dtype(dtype) &&
                      ldp >= heads * 2 * dim + (own ? kv_heads * (2 * dim + vdim) : 0) && (!own || (cache && slot_mapping)),
                  "diff_attn_prep: bad argument (heads=%d kv_heads=%d dim=%d vdim=%d ldp=%d)", heads, kv_heads, dim, vdim,
                  ldp);
  B200Q_CHECK_ARG(taps >= 0 && taps <= DIFF_MAX_TAPS && (taps == 0 || conv) && (taps <= 1 || state),
                  "diff_attn_prep: bad convolution (%d taps, at most %d)", taps, DIFF_MAX_TAPS);
  B200Q_CHECK_ARG(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim && (rot_dims == 0 || table),
                  "diff_attn_prep: rot_dims (%d) must be even and at most dim (%d)", rot_dims, dim);
  if (T_ == 0) return B200Q_OK;
  const bool tiled = b200q_diff_attn_tiled(dim, vdim, block_size, dtype);
  DiffPrep a{proj, bias, taps > 0 ? conv : nullptr, state, (const float2*)table, seq_desc, row_seq, slot_mapping, q, cache,
             slot_stride, tiled ? (float)(scale * 1.4426950408889634) : scale, ldp, heads, kv_heads, dim, vdim, taps,
             rot_dims, block_size, tiled ? 7 : 0, own ? 1 : 0};
  const int C = heads * 2 * dim + (own ? kv_heads * (2 * dim + vdim) : 0);
  cudaStream_t st = as_stream(stream);
  const bool v8 = tiled && taps <= 4 && ldp % 8 == 0 && slot_stride % 4 == 0 &&
                  ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(bias) | reinterpret_cast<uintptr_t>(conv) |
                    reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) &
                   15) == 0;
  if (v8) {
    dim3 grid(n_seqs, (C / 8 + 127) / 128, (longest_portion(max_portion, n_seqs, T_) + PREP_TOKENS - 1) / PREP_TOKENS);
    B200Q_CHECK_ARG(grid.y <= 65535 && grid.z <= 65535, "diff_attn_prep: step too large (%d tokens)", T_);
    if (taps <= 1) diff_prep_v8_kernel<1><<<grid, 128, 0, st>>>(a);
    else if (taps == 2) diff_prep_v8_kernel<2><<<grid, 128, 0, st>>>(a);
    else if (taps == 3) diff_prep_v8_kernel<3><<<grid, 128, 0, st>>>(a);
    else diff_prep_v8_kernel<4><<<grid, 128, 0, st>>>(a);
  } else {
    dim3 grid(T_, (C + 255) / 256);
    B200Q_CHECK_ARG(grid.y <= 65535, "diff_attn_prep: too many channels");
    if (tiled) diff_prep_kernel<bf16, bf16><<<grid, 256, 0, st>>>(a);
    else DISPATCH_T(dtype, (diff_prep_kernel<T, float><<<grid, 256, 0, st>>>(a)));
  }
  B200Q_LAUNCH_CHECK();
  if (taps > 1 && !(v8 && T_ == n_seqs)) {
    dim3 sgrid(n_seqs, (C + 255) / 256);
    DISPATCH_T(dtype, (diff_prep_state_kernel<T><<<sgrid, 256, 0, st>>>(a, v8 ? 1 : 0)));
    B200Q_LAUNCH_CHECK();
  }
  return B200Q_OK;
}

int b200q_diff_attn(const void* q, const void* cache, const int32_t* block_table, int bt_stride, const int32_t* row_seq,
                    const int32_t* positions, const int32_t* seq_desc, int n_seqs, int max_portion, int T_, int heads,
                    int kv_heads, int dim, int vdim, int block_size, const float* lambda, float mult, float eps, const void* gate, int ld_gate,
                    void* out, int ld_out, int dtype, void* stream) {
  B200Q_CHECK_ARG(q && cache && block_table && row_seq && positions && seq_desc && n_seqs > 0 && lambda && out &&
                      heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && dim <= 256 && vdim > 0 && vdim <= 512 &&
                      block_size > 0 && T_ >= 0 && eps >= 0.f && is_dtype(dtype) && (!gate || ld_gate >= heads) &&
                      ld_out >= heads * vdim,
                  "diff_attn: bad argument (heads=%d kv_heads=%d dim=%d (at most 256) vdim=%d (at most 512))", heads, kv_heads,
                  dim, vdim);
  if (T_ == 0) return B200Q_OK;
  int* failed = nullptr;
  if (!wait_flag(&failed)) {
    set_error("diff_attn: no mapped host memory");
    return B200Q_ECUDA;
  }
  const bool tiled = b200q_diff_attn_tiled(dim, vdim, block_size, dtype);
  DiffAttn a{q, cache, block_table, seq_desc, row_seq, positions, lambda, gate, out, failed, mult, eps, bt_stride, heads,
             kv_heads, dim, vdim, block_size, ld_gate, ld_out, tiled ? 7 : 0};
  cudaStream_t st = as_stream(stream);
  if (tiled) {
    B200Q_CHECK_ARG(((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15) == 0 &&
                        (reinterpret_cast<uintptr_t>(out) & 3) == 0 && ld_out % 2 == 0,
                    "diff_attn: queries and cache must be 16-byte aligned, output rows 4-byte aligned");
    const int longest = longest_portion(max_portion, n_seqs, T_);
    return dim <= 64 ? launch_diff_mma<64, 128>(a, n_seqs, longest, T_, st) : launch_diff_mma<128, 128>(a, n_seqs, longest, T_, st);
  }
  dim3 grid(T_, kv_heads, (heads / kv_heads + 3) / 4);
  B200Q_CHECK_ARG(grid.y <= 65535 && grid.z <= 65535, "diff_attn: too many heads");
  const size_t smem = (size_t)(8 * dim + 32 * (2 * dim + 1) + 32 * (vdim + 1)) * sizeof(float);
#define SCALAR(ACC)                                                                                                       \
  DISPATCH_T(dtype, {                                                                                                     \
    auto kern = diff_attn_kernel<T, ACC>;                                                                                 \
    if (smem > 48 * 1024) B200Q_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
    kern<<<grid, 256, smem, st>>>(a);                                                                                     \
  })
  if (vdim <= 64) SCALAR(2);
  else if (vdim <= 128) SCALAR(4);
  else if (vdim <= 256) SCALAR(8);
  else SCALAR(16);
#undef SCALAR
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

}  // extern "C"
