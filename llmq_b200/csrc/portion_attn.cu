// portion_attn.cu — softmax attention on the tensor cores (bf16 caches).  Prompt portions: 64 consecutive tokens of a
// sequence's portion and one head per CTA, keys in tiles of 64.  Two sources of keys and values share the kernel:
//   grouped-query attention   both from the paged cache ([kv_heads*dim | kv_heads*vdim] rows)
//   latent attention          the unrotated keys and the values as rows that were expanded from the cached latents for the
//                             sequence's visible span, the rotated key part from the paged cache.  A prompt reads every
//                             expanded row many times, so expanding it once costs less than carrying every query into the
//                             latent space (which single tokens do): per score dim + rot_dim + vdim products instead of
//                             2 kv_rank + rot_dim.
// Single tokens: one CTA per (sequence, key head), and per (token, 16 or 32 heads) in the latent space, below.
// Scores, softmax state and accumulators are fp32; queries and weights are rounded to bf16 as the products see them.
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
// keys lo .. pos0 + n - 1 are what a portion's tokens see
__device__ __forceinline__ int span_begin(const SeqView& s, int window) {
  return window > 0 ? max(0, s.pos0 - window + 1) : 0;
}

// 16 bytes into shared memory, zeros when `on` is false
__device__ __forceinline__ void cp_async16_zfill(void* dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}

// ------------------------------------------------------------------------------------------------
// the latents a step's portions see, gathered from their pages into dense rows (sequence by sequence, in order of the
// positions), and where each sequence's rows begin: span[s] = {first row, first position}.  CTA = 64 rows of a sequence.
// ------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) latent_gather_kernel(const bf16* __restrict__ cache, const int32_t* __restrict__ block_table,
                                                            int bt_stride, const int32_t* __restrict__ seq_desc, int window,
                                                            int bs_shift, int R, int RP, int cap, bf16* __restrict__ out,
                                                            int2* __restrict__ span) {
  __shared__ int part[8];
  const SeqView s = seq_view(seq_desc, blockIdx.x);
  if (s.n <= 1) return;
  int before = 0;
  for (int i = threadIdx.x; i < (int)blockIdx.x; i += 256) {
    const SeqView o = seq_view(seq_desc, i);
    if (o.n > 1) before += o.pos0 + o.n - span_begin(o, window);
  }
  before = __reduce_add_sync(0xffffffffu, before);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = before;
  __syncthreads();
  before = 0;
#pragma unroll
  for (int i = 0; i < 8; ++i) before += part[i];
  const int lo = span_begin(s, window), count = s.pos0 + s.n - lo;
  if (blockIdx.y == 0 && threadIdx.x == 0) span[blockIdx.x] = make_int2(before, lo);
  const int32_t* bt = block_table + (long long)blockIdx.x * bt_stride;
  const int per = R / 8, mask = (1 << bs_shift) - 1;
  for (int e = threadIdx.x; e < 64 * per; e += 256) {
    const int r = blockIdx.y * 64 + e / per, c = (e % per) * 8;
    if (r >= count || before + r >= cap) break;  // (the caller sizes `out` for all rows)
    const int pos = lo + r;
    const long long row = ((long long)bt[pos >> bs_shift] << bs_shift) + (pos & mask);
    st_v4(out + (long long)(before + r) * R + c, ld_v4(cache + row * RP + c));
  }
}

struct PortionAttn {
  const float* q32;   // grouped-query: [T, heads, dim], scale folded in; latent: [T, heads, kv_rank + rot_dim], rotated parts
  const bf16* q16;    // latent: rows of stride ldq, head h's unrotated query at h * (dim + rot_dim)
  const bf16* cache;  // paged rows of `row` elements
  const bf16 *kx, *vx;  // latent: expanded keys [rows][heads*dim] and values [rows][heads*vdim]
  const int2* span;
  const int32_t *block_table, *seq_desc;
  const float* sink;
  const bf16* gate;
  bf16* out;  // [T, heads*vdim]
  float qmul;         // what turns a stored query into one whose scores are in base 2
  int bt_stride, heads, kv_heads, dim, rot_dim, kv_rank, row, ldq, bs_shift, window, ld_gate, channel_gate, skip_single;
};

// ------------------------------------------------------------------------------------------------
// 4 warps of 16 tokens; a tile's rows lie in shared memory with their 16-byte pieces permuted (piece ^ (row & 7)), so
// ldmatrix meets no bank conflicts without padding.  Eight threads copy 128 bytes of a row side by side; the page
// numbers of the tile after the next are read one tile ahead.  Late tokens (the longest rows) are launched first.
// ------------------------------------------------------------------------------------------------
constexpr int PATT_KEYS = 64;
constexpr float PATT_NEG = -1e30f;  // finite floor of the running maximum: exp2(masked - floor) = 0, never NaN
template <int DK, int DV, bool LATENT>
__global__ void __launch_bounds__(128, 2) portion_attn_kernel(const PortionAttn a) {
  extern __shared__ __align__(128) uint8_t smraw[];
  bf16* kbuf = reinterpret_cast<bf16*>(smraw);      // [2][64][DK]
  bf16* vbuf = kbuf + 2 * PATT_KEYS * DK;           // [2][64][DV]
  const SeqView sq = seq_view(a.seq_desc, blockIdx.x);
  const int r0 = (gridDim.z - 1 - blockIdx.z) * 64;
  if (r0 >= sq.n || (a.skip_single && sq.n == 1)) return;
  const int nrows = min(64, sq.n - r0), h = blockIdx.y, g = h / (a.heads / a.kv_heads);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, q4 = lane & 3;
  const int p_first = sq.pos0 + r0, p_last = p_first + nrows - 1;
  const int lo = a.window > 0 ? max(0, p_first - a.window + 1) : 0;
  const int ntiles = (p_last - lo) / PATT_KEYS + 1;
  const int32_t* bt = a.block_table + (long long)blockIdx.x * a.bt_stride;
  const int page_mask = (1 << a.bs_shift) - 1;
  int2 sp = make_int2(0, 0);
  if (LATENT) sp = a.span[blockIdx.x];
  // this thread copies pieces (tid & 7), + 8, ... of rows tid / 8 + 16 i of a tile
  const int cr = tid >> 3, cc = tid & 7;
  int page[4];
  auto look_up = [&](int c) {
#pragma unroll
    for (int i = 0; i < 4; ++i) page[i] = bt[min(lo + c * PATT_KEYS + cr + 16 * i, p_last) >> a.bs_shift];
  };
  auto load_tile = [&](int c, int buf) {
    bf16* kb = kbuf + buf * PATT_KEYS * DK;
    bf16* vb = vbuf + buf * PATT_KEYS * DV;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = cr + 16 * i, j = lo + c * PATT_KEYS + r, pos = min(j, p_last);
      const bool on = j <= p_last;  // rows behind the last token are zeros
      const bf16* row = a.cache + (((long long)page[i] << a.bs_shift) + (pos & page_mask)) * a.row;
      const bf16 *k0, *k1 = nullptr, *v0;
      if (LATENT) {
        const long long x = sp.x + (pos - sp.y);
        k0 = a.kx + (x * a.heads + h) * a.dim;
        k1 = row + a.kv_rank - a.dim;  // rotated part: columns dim .. DK - 1 of the key
        v0 = a.vx + (x * a.heads + h) * DV;
      } else {
        k0 = row + g * DK;
        v0 = row + a.kv_heads * DK + g * DV;
      }
#pragma unroll
      for (int k = 0; k < DK / 64; ++k) {
        const int p = cc + 8 * k;
        cp_async16_zfill(kb + r * DK + ((p ^ (r & 7)) << 3), (LATENT && p * 8 >= a.dim ? k1 : k0) + p * 8, on);
      }
#pragma unroll
      for (int k = 0; k < DV / 64; ++k) {
        const int p = cc + 8 * k;
        cp_async16_zfill(vb + r * DV + ((p ^ (r & 7)) << 3), v0 + p * 8, on);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // queries into the second key buffer, then into registers; rows past the portion are zeros
  look_up(0);
  load_tile(0, 0);
  {
    bf16* qb = kbuf + PATT_KEYS * DK;
    for (int e = tid; e < 64 * (DK / 8); e += 128) {
      const int r = e / (DK / 8), p = e % (DK / 8);
      uint4 w = make_uint4(0, 0, 0, 0);
      if (r < nrows) {
        const long long th = (long long)(sq.row0 + r0 + r) * a.heads + h;
        float v[8];
        if (LATENT && p * 8 < a.dim) {
          const uint4 x = ld_v4(a.q16 + (long long)(sq.row0 + r0 + r) * a.ldq + (long long)h * (a.dim + a.rot_dim) + p * 8);
          const uint32_t xw[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            v[2 * i] = bf16_lo(xw[i]);
            v[2 * i + 1] = bf16_hi(xw[i]);
          }
        } else {
          const float* src = LATENT ? a.q32 + th * (a.kv_rank + a.rot_dim) + a.kv_rank + p * 8 - a.dim : a.q32 + th * DK + p * 8;
          const float4 x = *reinterpret_cast<const float4*>(src), y = *reinterpret_cast<const float4*>(src + 4);
          v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
          v[4] = y.x; v[5] = y.y; v[6] = y.z; v[7] = y.w;
        }
        w = make_uint4(pack_bf16x2(v[0] * a.qmul, v[1] * a.qmul), pack_bf16x2(v[2] * a.qmul, v[3] * a.qmul),
                       pack_bf16x2(v[4] * a.qmul, v[5] * a.qmul), pack_bf16x2(v[6] * a.qmul, v[7] * a.qmul));
      }
      st_v4(qb + r * DK + ((p ^ (r & 7)) << 3), w);
    }
  }
  __syncthreads();
  const int swz = lane & 7;
  uint32_t qf[DK / 16][4];
  {
    const uint32_t q_s = smem_u32(kbuf + PATT_KEYS * DK + (warp * 16 + (lane & 15)) * DK);
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks)
      ldsm_x4(q_s + (uint32_t)(((ks * 2 + (lane >> 4)) ^ swz) << 4), qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3]);
  }
  const int krow = (lane & 7) + 8 * (lane >> 4), kck = (lane >> 3) & 1;
  const int vrow = ((lane >> 3) & 1) * 8 + (lane & 7), vck = lane >> 4;
  int p_row[2], lo_row[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int i = warp * 16 + gq + 8 * r;
    p_row[r] = i < nrows ? p_first + i : -1;  // a dead row sees no key
    lo_row[r] = a.window > 0 ? p_row[r] - a.window + 1 : 0;
  }
  const int w_first = p_first + warp * 16, w_last = min(w_first + 15, p_last);
  const int w_lo = a.window > 0 ? w_last - a.window + 1 : 0;  // first key that the warp's last token sees
  const bool warp_live = warp * 16 < nrows;
  float m_[2] = {PATT_NEG, PATT_NEG}, l_[2] = {0.f, 0.f};
  if (a.sink) {  // counted once per row: by the first of the four threads that share it
    m_[0] = m_[1] = a.sink[h] * 1.4426950408889634f;
    if (q4 == 0) l_[0] = l_[1] = 1.f;
  }
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  if (ntiles > 1) look_up(1);
  for (int c = 0; c < ntiles; ++c) {
    const int buf = c & 1, j0 = lo + c * PATT_KEYS;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // tile c is whole for everyone, tile c - 1 (first time: the queries) is done with
    if (c + 1 < ntiles) {
      load_tile(c + 1, buf ^ 1);
      if (c + 2 < ntiles) look_up(c + 2);
    }
    if (!warp_live || j0 > w_last || (a.window > 0 && j0 + PATT_KEYS - 1 < w_first - a.window + 1)) continue;
    const uint32_t kb_s = smem_u32(kbuf + buf * PATT_KEYS * DK), vb_s = smem_u32(vbuf + buf * PATT_KEYS * DV);
    float s[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      const uint32_t kp = kb_s + (uint32_t)(krow * DK * 2) + (uint32_t)(((ks * 2 + kck) ^ swz) << 4);
#pragma unroll
      for (int nt2 = 0; nt2 < 4; ++nt2) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4(kp + (uint32_t)(nt2 * 16 * DK * 2), b0, b1, b2, b3);
        mma_bf16_16816(s[2 * nt2], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b0, b1);
        mma_bf16_16816(s[2 * nt2 + 1], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b2, b3);
      }
    }
    if (j0 + PATT_KEYS - 1 > w_first || nrows < 64 || j0 < w_lo) {
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = j0 + nt * 8 + 2 * q4 + (e & 1);
          if (j > p_row[e >> 1] || j < lo_row[e >> 1]) s[nt][e] = -INFINITY;
        }
    }
    uint32_t pk[16];
    float corr[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float mx = PATT_NEG;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) mx = fmaxf(mx, fmaxf(s[nt][2 * r], s[nt][2 * r + 1]));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float mn = fmaxf(m_[r], mx);
      corr[r] = exp2f(m_[r] - mn);
      m_[r] = mn;
      float ps = 0.f;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        const uint32_t v = pack_bf16x2(exp2f(s[nt][2 * r] - mn), exp2f(s[nt][2 * r + 1] - mn));  // masked: exp2(-inf) = 0
        ps += bf16_lo(v) + bf16_hi(v);
        pk[(nt >> 1) * 4 + (nt & 1) * 2 + r] = v;
      }
      l_[r] = l_[r] * corr[r] + ps;
    }
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int i = 0; i < DV / 8; ++i) {
        o[i][0] *= corr[0];
        o[i][1] *= corr[0];
        o[i][2] *= corr[1];
        o[i][3] *= corr[1];
      }
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      const uint32_t vp = vb_s + (uint32_t)((kk * 16 + vrow) * DV * 2);
#pragma unroll
      for (int nd = 0; nd < DV / 16; ++nd) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4_t(vp + (uint32_t)(((nd * 2 + vck) ^ swz) << 4), b0, b1, b2, b3);
        mma_bf16_16816(o[2 * nd], pk[4 * kk], pk[4 * kk + 1], pk[4 * kk + 2], pk[4 * kk + 3], b0, b1);
        mma_bf16_16816(o[2 * nd + 1], pk[4 * kk], pk[4 * kk + 1], pk[4 * kk + 2], pk[4 * kk + 3], b2, b3);
      }
    }
  }
  if (!warp_live) return;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float l = l_[r];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    if (p_row[r] < 0) continue;
    const long long t = sq.row0 + (p_row[r] - sq.pos0);
    const float gv = a.gate && !a.channel_gate ? sigmoidf_(__bfloat162float(a.gate[t * a.ld_gate + h])) : 1.f;
    const float inv = gv / l;
    bf16* orow = a.out + (t * a.heads + h) * DV;
    const bf16* grow = a.channel_gate ? a.gate + t * a.ld_gate + (long long)h * DV : nullptr;
#pragma unroll
    for (int nt = 0; nt < DV / 8; ++nt) {
      const int d = nt * 8 + 2 * q4;
      float g0 = 1.f, g1 = 1.f;
      if (grow) {
        g0 = sigmoidf_(__bfloat162float(grow[d]));
        g1 = sigmoidf_(__bfloat162float(grow[d + 1]));
      }
      *reinterpret_cast<uint32_t*>(orow + d) = pack_bf16x2(o[nt][2 * r] * inv * g0, o[nt][2 * r + 1] * inv * g1);
    }
  }
}

// ------------------------------------------------------------------------------------------------
// single decoded tokens, grouped-query attention: one CTA per (sequence, key head); the 16 rows of a tile are the heads of
// the group.  Each warp takes the tiles of 16 keys warp, warp + nw, ... through its own ring of STG stages (no CTA barrier in
// the loop), the rows of a stage looked up one tile before they are asked for; the warps' states are merged in a fixed
// order.  nw (2, 4 or 8) is the block's size: many sequences take small blocks, which fit one wave with four per SM.
// ------------------------------------------------------------------------------------------------
constexpr int TATT_KEYS = 16, TATT_STG = 3;
template <int DK, int DV>
__global__ void __launch_bounds__(256) token_attn_kernel(const PortionAttn a) {
  extern __shared__ __align__(128) uint8_t smraw[];
  constexpr int STAGE = TATT_KEYS * (DK + DV);       // elements of a stage: keys, then values
  constexpr int MS = DV + 2;
  const SeqView sq = seq_view(a.seq_desc, blockIdx.x);
  if (sq.n != 1) return;  // portions of prompts take the tile kernel
  const int nw = blockDim.x >> 5, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, q4 = lane & 3;
  const int g = blockIdx.y, rep = a.heads / a.kv_heads;
  bf16* ring = reinterpret_cast<bf16*>(smraw) + (long long)warp * TATT_STG * STAGE;
  bf16* qb = reinterpret_cast<bf16*>(smraw) + (long long)nw * TATT_STG * STAGE;  // [16][DK]
  float* mrg = reinterpret_cast<float*>(smraw);                                  // after the loop: [nw][16][DV + 2]
  const int p = sq.pos0, lo = a.window > 0 ? max(0, p - a.window + 1) : 0;
  const int ntiles = (p - lo) / TATT_KEYS + 1, n_it = warp < ntiles ? (ntiles - warp + nw - 1) / nw : 0;
  const long long t = sq.row0;
  const int32_t* bt = a.block_table + (long long)blockIdx.x * a.bt_stride;
  const int page_mask = (1 << a.bs_shift) - 1;
  int row_next = 0;  // lane l (mod 16): cache row of key l of the next tile to be asked for
  auto look_up = [&](int it) {
    const int pos = min(lo + (warp + it * nw) * TATT_KEYS + (lane & 15), p);
    row_next = (bt[pos >> a.bs_shift] << a.bs_shift) + (pos & page_mask);
  };
  auto load_tile = [&](int it) {
    bf16* kb = ring + (it % TATT_STG) * STAGE;
    const int j0 = lo + (warp + it * nw) * TATT_KEYS;
    constexpr int PER = (DK + DV) / 8;  // 16-byte pieces of a key and its value
#pragma unroll
    for (int i = 0; i < TATT_KEYS * PER / 32; ++i) {
      const int e = i * 32 + lane, j = e / PER, c = e % PER;
      const bf16* row = a.cache + (long long)__shfl_sync(0xffffffffu, row_next, j) * a.row;
      const bool key = c < DK / 8;
      const int v = c - DK / 8;
      const bf16* src = key ? row + g * DK + c * 8 : row + a.kv_heads * DK + g * DV + v * 8;
      bf16* dst = key ? kb + j * DK + ((c ^ (j & 7)) << 3) : kb + TATT_KEYS * DK + j * DV + ((v ^ (j & 7)) << 3);
      cp_async16_zfill(dst, src, j0 + j <= p);
    }
  };
  auto commit = [&]() { asm volatile("cp.async.commit_group;" ::: "memory"); };
  if (n_it > 0) look_up(0);
  for (int i = 0; i < TATT_STG - 1; ++i) {  // every turn commits a group, so that the count of groups is the same for all
    if (i < n_it) {
      load_tile(i);
      if (i + 1 < n_it) look_up(i + 1);
    }
    commit();
  }
  for (int e = tid; e < 16 * (DK / 8); e += blockDim.x) {
    const int r = e / (DK / 8), c = e % (DK / 8);
    uint4 w = make_uint4(0, 0, 0, 0);
    if (r < rep) {
      const float* src = a.q32 + (t * a.heads + g * rep + r) * DK + c * 8;
      const float4 x = *reinterpret_cast<const float4*>(src), y = *reinterpret_cast<const float4*>(src + 4);
      w = make_uint4(pack_bf16x2(x.x * a.qmul, x.y * a.qmul), pack_bf16x2(x.z * a.qmul, x.w * a.qmul),
                     pack_bf16x2(y.x * a.qmul, y.y * a.qmul), pack_bf16x2(y.z * a.qmul, y.w * a.qmul));
    }
    st_v4(qb + r * DK + ((c ^ (r & 7)) << 3), w);
  }
  __syncthreads();
  const int swz = lane & 7;
  uint32_t qf[DK / 16][4];
  {
    const uint32_t q_s = smem_u32(qb + (lane & 15) * DK);
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks)
      ldsm_x4(q_s + (uint32_t)(((ks * 2 + (lane >> 4)) ^ swz) << 4), qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3]);
  }
  const int krow = (lane & 7) + 8 * (lane >> 4), kck = (lane >> 3) & 1;
  const int vrow = ((lane >> 3) & 1) * 8 + (lane & 7), vck = lane >> 4;
  float m_[2] = {PATT_NEG, PATT_NEG}, l_[2] = {0.f, 0.f};
  if (a.sink && warp == 0) {  // counted once: by the first warp's state, there by the first of a row's four threads
#pragma unroll
    for (int r = 0; r < 2; ++r)
      if (gq + 8 * r < rep) {
        m_[r] = a.sink[g * rep + gq + 8 * r] * 1.4426950408889634f;
        l_[r] = q4 == 0 ? 1.f : 0.f;
      }
  }
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  for (int it = 0; it < n_it; ++it) {
    asm volatile("cp.async.wait_group %0;" ::"n"(TATT_STG - 2) : "memory");
    __syncwarp();  // tile `it` is whole for the warp; the stage of tile it - 1 is done with
    if (it + TATT_STG - 1 < n_it) {
      load_tile(it + TATT_STG - 1);
      if (it + TATT_STG < n_it) look_up(it + TATT_STG);
    }
    commit();
    const bf16* kb = ring + (it % TATT_STG) * STAGE;
    const uint32_t kb_s = smem_u32(kb), vb_s = smem_u32(kb + TATT_KEYS * DK);
    const int j0 = lo + (warp + it * nw) * TATT_KEYS;
    float s[2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4(kb_s + (uint32_t)(krow * DK * 2) + (uint32_t)(((ks * 2 + kck) ^ swz) << 4), b0, b1, b2, b3);
      mma_bf16_16816(s[0], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b0, b1);
      mma_bf16_16816(s[1], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b2, b3);
    }
    uint32_t pk[4];
    float corr[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float mx = PATT_NEG;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          if (gq + 8 * r >= rep || j0 + nt * 8 + 2 * q4 + k > p) s[nt][2 * r + k] = -INFINITY;
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
      for (int i = 0; i < DV / 8; ++i) {
        o[i][0] *= corr[0];
        o[i][1] *= corr[0];
        o[i][2] *= corr[1];
        o[i][3] *= corr[1];
      }
    }
    const uint32_t vp = vb_s + (uint32_t)(vrow * DV * 2);
#pragma unroll
    for (int nd = 0; nd < DV / 16; ++nd) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4_t(vp + (uint32_t)(((nd * 2 + vck) ^ swz) << 4), b0, b1, b2, b3);
      mma_bf16_16816(o[2 * nd], pk[0], pk[1], pk[2], pk[3], b0, b1);
      mma_bf16_16816(o[2 * nd + 1], pk[0], pk[1], pk[2], pk[3], b2, b3);
    }
    __syncwarp();  // every lane is done with the stage before its next rows are asked for
  }
  // ---- merge: [warp][row][DV + 2] = (o..., m, l); a warp without tiles holds (0, floor, 0) ----
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();  // every warp is done with its ring: it becomes the merge area
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_[r] += __shfl_xor_sync(0xffffffffu, l_[r], 1);
    l_[r] += __shfl_xor_sync(0xffffffffu, l_[r], 2);
    float* dst = mrg + (long long)(warp * 16 + gq + 8 * r) * MS;
#pragma unroll
    for (int nt = 0; nt < DV / 8; ++nt) {
      dst[nt * 8 + 2 * q4] = o[nt][2 * r];
      dst[nt * 8 + 2 * q4 + 1] = o[nt][2 * r + 1];
    }
    if (q4 == 0) {
      dst[DV] = m_[r];
      dst[DV + 1] = l_[r];
    }
  }
  __syncthreads();
  for (int hh = warp; hh < rep; hh += nw) {  // one warp per head
    float mx = PATT_NEG, den = 0.f;
    for (int w = 0; w < nw; ++w) mx = fmaxf(mx, mrg[(long long)(w * 16 + hh) * MS + DV]);
    for (int w = 0; w < nw; ++w) den = fmaf(mrg[(long long)(w * 16 + hh) * MS + DV + 1], exp2f(mrg[(long long)(w * 16 + hh) * MS + DV] - mx), den);
    const int h = g * rep + hh;
    const float gv = a.gate && !a.channel_gate ? sigmoidf_(__bfloat162float(a.gate[t * a.ld_gate + h])) : 1.f;
    const float inv = gv / den;
#pragma unroll
    for (int i = 0; i < DV / 32; ++i) {
      const int d = lane + 32 * i;
      float num = 0.f;
      for (int w = 0; w < nw; ++w) num = fmaf(mrg[(long long)(w * 16 + hh) * MS + d], exp2f(mrg[(long long)(w * 16 + hh) * MS + DV] - mx), num);
      if (a.channel_gate) num *= sigmoidf_(__bfloat162float(a.gate[t * a.ld_gate + (long long)h * DV + d]));
      a.out[(t * a.heads + h) * DV + d] = __float2bfloat16_rn(num * inv);
    }
  }
}

// ------------------------------------------------------------------------------------------------
// latent attention in the latent space (single tokens, and portions that are not worth expanding): one CTA of 8 warps per
// (token, MT * 16 heads).  A cached row [latent | rotated part] serves all of the CTA's heads as key and, its latent, as value.
// Chunks of CH = 64 / MT keys pass through a ring of STG stages, a row = one bulk copy (the warps ask
// for an eighth of a chunk each: a warp's lanes issue their copies one after the other).  Every warp scores one 16 x 8 tile of (heads, keys) over all
// kv_rank + rot_dim dimensions (queries as bf16 high and low parts, read from shared memory), the scores meet in shared
// memory, and every warp accumulates kv_rank / 8 of the latent dimensions.  Chunks start at the token's first visible key, so
// its arithmetic does not depend on how the prompt was cut.  Needs kv_rank a multiple of 128 up to 512.
// ------------------------------------------------------------------------------------------------
struct LatentTokens {
  const float* qa;    // [T, heads, RP]
  const bf16* cache;  // paged rows of RP elements
  const int32_t *block_table, *row_seq, *positions;
  const float* sink;
  const bf16* gate;
  bf16* out;  // [T, heads, R]
  int* failed;  // set when a bounded wait runs out
  float scale;  // of the scores, in base 2
  int bt_stride, heads, R, RP, bs_shift, window, ld_gate;
};
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <int MT, int NT>  // NT: 8-wide tiles of latent dimensions per warp
__global__ void __launch_bounds__(256, 1) latent_token_kernel(const LatentTokens a) {
  constexpr int CH = 64 / MT, STG = MT == 1 ? 2 : 3, SLD = CH + 4, NK = CH / 8;
  extern __shared__ __align__(128) uint8_t smraw[];
  __shared__ __align__(8) uint64_t full[STG];
  const int LDS = a.RP + 8;  // padded rows: ldmatrix rows fall on different banks
  bf16* ring = reinterpret_cast<bf16*>(smraw);                   // [STG][CH][LDS]
  bf16* qhi = ring + STG * CH * LDS;                             // [MT*16][LDS]
  bf16* qlo = qhi + MT * 16 * LDS;                               // [MT*16][LDS]
  float* sc = reinterpret_cast<float*>(qlo + MT * 16 * LDS);     // [MT*16][SLD]
  const int t = blockIdx.x, h0 = blockIdx.y * MT * 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, q4 = lane & 3;
  const int p = a.positions[t], lo = a.window > 0 ? max(0, p - a.window + 1) : 0;
  const int nchunks = (p - lo) / CH + 1;
  const int32_t* bt = a.block_table + (long long)a.row_seq[t] * a.bt_stride;
  const int page_mask = (1 << a.bs_shift) - 1;
  // lanes l < CH / 8 of warp w ask for key w * CH / 8 + l of a chunk; row_next: its cache row in the next chunk to be asked for
  const int key_of = warp * (CH / 8) + (lane & (CH / 8 - 1));
  int row_next = 0;
  auto look_up = [&](int c) {
    const int pos = min(lo + c * CH + key_of, p);
    row_next = (bt[pos >> a.bs_shift] << a.bs_shift) + (pos & page_mask);
  };
  auto load_chunk = [&](int c) {
    const int stage = c % STG, n = min(CH, p + 1 - (lo + c * CH));
    if (tid == 0) mbar_expect_tx(full + stage, (uint32_t)(n * a.RP * 2));  // (copies that land first wait for it)
    if (lane < CH / 8 && key_of < n)
      tma_bulk_g2s(ring + (stage * CH + key_of) * LDS, a.cache + (long long)row_next * a.RP, (uint32_t)(a.RP * 2), full + stage);
    __syncwarp();
  };
  look_up(0);
  if (tid == 0) {
#pragma unroll
    for (int i = 0; i < STG; ++i) mbar_init(full + i, 1);
    mbar_fence_init();
  }
  __syncthreads();  // the barriers are there
#pragma unroll
  for (int c = 0; c < STG - 1; ++c)
    if (c < nchunks) {
      load_chunk(c);
      if (c + 1 < nchunks) look_up(c + 1);
    }
  for (int e = tid; e < MT * 16 * (a.RP / 4); e += 256) {
    const int r = e / (a.RP / 4), d = (e % (a.RP / 4)) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (h0 + r < a.heads) v = *reinterpret_cast<const float4*>(a.qa + ((long long)t * a.heads + h0 + r) * a.RP + d);
    const float x[4] = {v.x * a.scale, v.y * a.scale, v.z * a.scale, v.w * a.scale};
    const uint32_t w0 = pack_bf16x2(x[0], x[1]), w1 = pack_bf16x2(x[2], x[3]);
    *reinterpret_cast<uint2*>(qhi + r * LDS + d) = make_uint2(w0, w1);
    *reinterpret_cast<uint2*>(qlo + r * LDS + d) =
        make_uint2(pack_bf16x2(x[0] - bf16_lo(w0), x[1] - bf16_hi(w0)), pack_bf16x2(x[2] - bf16_lo(w1), x[3] - bf16_hi(w1)));
  }
  const int mt = warp / NK, nk = warp % NK;  // the score tile of this warp
  const uint32_t a_off = (uint32_t)(((mt * 16 + (lane & 15)) * LDS + (lane >> 4) * 8) * 2);
  const uint32_t qhi_s = smem_u32(qhi) + a_off, qlo_s = smem_u32(qlo) + a_off;
  const uint32_t k_off = (uint32_t)(((nk * 8 + (lane & 7)) * LDS + 8 * (lane >> 3)) * 2);  // 8 keys x 32 dimensions
  const int dim_w = warp * NT * 8;
  float m_[MT][2], l_[MT][2], o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int h = h0 + m * 16 + gq + 8 * r;
      const bool on = a.sink && h < a.heads;  // every thread holds its rows' whole sums: the sink's 1 belongs to each
      m_[m][r] = on ? a.sink[h] * 1.4426950408889634f : -INFINITY;
      l_[m][r] = on ? 1.f : 0.f;
    }
#pragma unroll
    for (int i = 0; i < NT; ++i) o[m][i][0] = o[m][i][1] = o[m][i][2] = o[m][i][3] = 0.f;
  }
  for (int c = 0; c < nchunks; ++c) {
    const int n = min(CH, p + 1 - (lo + c * CH));
    bool ok = mbar_wait_limited(full + c % STG, (uint32_t)(c / STG) & 1u);
    if (n < CH)  // rows behind the last key: their weights are zeros, their values must not be NaNs
      for (int e = tid; e < (CH - n) * (a.R / 8); e += 256)
        st_v4(ring + ((c % STG) * CH + n + e / (a.R / 8)) * LDS + (e % (a.R / 8)) * 8, make_uint4(0, 0, 0, 0));
    ok = __syncthreads_and(ok);  // chunk c (and, first time, the queries) is there; chunk c - 1 and its scores are done with
    if (!ok) {  // give up: let the copies already on their way land first
      if (tid == 0) {
        for (int i = c + 1; i < c + STG - 1 && i < nchunks; ++i) mbar_wait_limited(full + i % STG, (uint32_t)(i / STG) & 1u);
        *(volatile int*)a.failed = 1;
      }
      return;
    }
    if (c + STG - 1 < nchunks) {
      load_chunk(c + STG - 1);
      if (c + STG < nchunks) look_up(c + STG);
    }
    const uint32_t kb_s = smem_u32(ring + (c % STG) * CH * LDS);
    {
      float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f}, u0[4] = {0.f, 0.f, 0.f, 0.f}, u1[4] = {0.f, 0.f, 0.f, 0.f};
      int d = 0;
#pragma unroll 3
      for (; d + 32 <= a.RP; d += 32) {
        uint32_t b0, b1, b2, b3, h0_, h1, h2, h3, g0, g1, g2, g3;
        ldsm_x4(kb_s + k_off + d * 2, b0, b1, b2, b3);
        ldsm_x4(qhi_s + d * 2, h0_, h1, h2, h3);
        ldsm_x4(qlo_s + d * 2, g0, g1, g2, g3);
        mma_bf16_16816(s0, h0_, h1, h2, h3, b0, b1);
        mma_bf16_16816(u0, g0, g1, g2, g3, b0, b1);
        ldsm_x4(qhi_s + d * 2 + 32, h0_, h1, h2, h3);
        ldsm_x4(qlo_s + d * 2 + 32, g0, g1, g2, g3);
        mma_bf16_16816(s1, h0_, h1, h2, h3, b2, b3);
        mma_bf16_16816(u1, g0, g1, g2, g3, b2, b3);
      }
      if (d < a.RP) {  // 16 dimensions left
        uint32_t b0, b1, b2, b3, h0_, h1, h2, h3;
        ldsm_x4(kb_s + k_off + d * 2 - 32, b0, b1, b2, b3);  // (from 16 before: the last 32 of the row)
        ldsm_x4(qhi_s + d * 2, h0_, h1, h2, h3);
        mma_bf16_16816(s0, h0_, h1, h2, h3, b2, b3);
        ldsm_x4(qlo_s + d * 2, h0_, h1, h2, h3);
        mma_bf16_16816(u0, h0_, h1, h2, h3, b2, b3);
      }
      float* dst = sc + (mt * 16 + gq) * SLD + nk * 8 + 2 * q4;
      *reinterpret_cast<float2*>(dst) = make_float2((s0[0] + s1[0]) + (u0[0] + u1[0]), (s0[1] + s1[1]) + (u0[1] + u1[1]));
      *reinterpret_cast<float2*>(dst + 8 * SLD) = make_float2((s0[2] + s1[2]) + (u0[2] + u1[2]), (s0[3] + s1[3]) + (u0[3] + u1[3]));
    }
    __syncthreads();
    uint32_t pk[MT][NK * 2];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      float corr[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float* src = sc + (m * 16 + gq + 8 * r) * SLD + 2 * q4;
        float v[NK * 2], mx = -INFINITY;
#pragma unroll
        for (int k = 0; k < NK; ++k) {
          const float2 x = *reinterpret_cast<const float2*>(src + 8 * k);
          v[2 * k] = x.x;
          v[2 * k + 1] = x.y;
        }
        if (n < CH) {
#pragma unroll
          for (int k = 0; k < NK * 2; ++k)
            if ((k >> 1) * 8 + 2 * q4 + (k & 1) >= n) v[k] = -INFINITY;
        }
#pragma unroll
        for (int k = 0; k < NK * 2; ++k) mx = fmaxf(mx, v[k]);
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float mn = fmaxf(m_[m][r], mx);
        corr[r] = ex2(m_[m][r] - mn);
        m_[m][r] = mn;
        float ps = 0.f;
#pragma unroll
        for (int k = 0; k < NK; ++k) {
          // rounded to what the value product sees (bf16), so that a row's weights still add up to one
          const uint32_t w = pack_bf16x2(ex2(v[2 * k] - mn), ex2(v[2 * k + 1] - mn));
          ps += bf16_lo(w) + bf16_hi(w);
          pk[m][(k >> 1) * 4 + (k & 1) * 2 + r] = w;
        }
        ps += __shfl_xor_sync(0xffffffffu, ps, 1);
        ps += __shfl_xor_sync(0xffffffffu, ps, 2);
        l_[m][r] = l_[m][r] * corr[r] + ps;
      }
      if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          o[m][i][0] *= corr[0];
          o[m][i][1] *= corr[0];
          o[m][i][2] *= corr[1];
          o[m][i][3] *= corr[1];
        }
      }
    }
#pragma unroll
    for (int kk = 0; kk < CH / 16; ++kk) {
      const int key = kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
      const uint32_t v_row = kb_s + (uint32_t)((key * LDS + dim_w + 8 * (lane >> 4)) * 2);
#pragma unroll
      for (int nd = 0; nd < NT / 2; ++nd) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4_t(v_row + nd * 32, b0, b1, b2, b3);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16_16816(o[m][2 * nd], pk[m][4 * kk], pk[m][4 * kk + 1], pk[m][4 * kk + 2], pk[m][4 * kk + 3], b0, b1);
          mma_bf16_16816(o[m][2 * nd + 1], pk[m][4 * kk], pk[m][4 * kk + 1], pk[m][4 * kk + 2], pk[m][4 * kk + 3], b2, b3);
        }
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int h = h0 + m * 16 + gq + 8 * r;
      if (h >= a.heads) continue;
      const float inv = (a.gate ? sigmoidf_(__bfloat162float(a.gate[(long long)t * a.ld_gate + h])) : 1.f) / l_[m][r];
      bf16* orow = a.out + ((long long)t * a.heads + h) * a.R + dim_w + 2 * q4;
#pragma unroll
      for (int i = 0; i < NT; ++i)
        *reinterpret_cast<uint32_t*>(orow + i * 8) = pack_bf16x2(o[m][i][2 * r] * inv, o[m][i][2 * r + 1] * inv);
    }
}

template <int MT, int NT>
static int launch_latent_tokens(const LatentTokens& a, int T, cudaStream_t st) {
  constexpr int CH = 64 / MT, STG = MT == 1 ? 2 : 3;
  const int smem = ((STG * CH + 2 * MT * 16) * (a.RP + 8)) * 2 + MT * 16 * (CH + 4) * 4;
  auto kern = latent_token_kernel<MT, NT>;
  B200Q_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  kern<<<dim3(T, (a.heads + MT * 16 - 1) / (MT * 16)), 256, smem, st>>>(a);
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

static int shift_of(int block_size) {  // -1: not a power of two
  int s = 0;
  while ((1 << s) < block_size) ++s;
  return (1 << s) == block_size ? s : -1;
}

template <int DK, int DV, bool LATENT>
static int launch_portions(const PortionAttn& a, int n_seqs, int longest, cudaStream_t st) {
  dim3 grid(n_seqs, a.heads, (longest + 63) / 64);
  B200Q_CHECK_ARG(grid.y <= 65535 && grid.z <= 65535, "portion_attn: step too large (portions of %d tokens)", longest);
  constexpr int smem = 2 * PATT_KEYS * (DK + DV) * 2;
  auto kern = portion_attn_kernel<DK, DV, LATENT>;
  B200Q_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  kern<<<grid, 128, smem, st>>>(a);
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

template <int DK, int DV>
static int launch_gqa_portions(const PortionAttn& a, int n_seqs, int longest, cudaStream_t st) {
  return launch_portions<DK, DV, false>(a, n_seqs, longest, st);
}

template <int DK, int DV>
static int launch_tokens(const PortionAttn& a, int n_seqs, cudaStream_t st) {
  const long long blocks = (long long)n_seqs * a.kv_heads;
  const int nw = blocks > 2 * 148 ? 2 : blocks > 148 ? 4 : 8;
  const int smem = std::max(nw * TATT_STG * TATT_KEYS * (DK + DV) * 2 + 16 * DK * 2, nw * 16 * (DV + 2) * 4);
  auto kern = token_attn_kernel<DK, DV>;
  B200Q_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  kern<<<dim3(n_seqs, a.kv_heads), nw * 32, smem, st>>>(a);
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

static bool portion_attn_on() {  // B200Q_PORTION_ATTN=0: the kernels it replaces
  static const bool on = [] {
    const char* v = getenv("B200Q_PORTION_ATTN");
    return !v || atoi(v) != 0;
  }();
  return on;
}

bool latent_tokens_ok(const float* qa, const void* cache, const void* out, int R, int P, int block_size) {
  return portion_attn_on() && (R == 128 || R == 256 || R == 384 || R == 512) && P >= 0 && P <= 64 && P % 16 == 0 &&
         shift_of(block_size) >= 0 &&
         ((reinterpret_cast<uintptr_t>(qa) | reinterpret_cast<uintptr_t>(cache)) & 15) == 0 &&
         (reinterpret_cast<uintptr_t>(out) & 3) == 0;
}

int latent_tokens(const float* qa, const void* cache, const int32_t* block_table, int bt_stride, const int32_t* row_seq,
                  const int32_t* positions, int T, int heads, int R, int P, int block_size, int window, float scale,
                  const float* sink, const void* gate, int ld_gate, void* out, cudaStream_t st) {
  int* failed = nullptr;
  if (!wait_flag(&failed)) {
    set_error("latent_attn: no mapped host memory");
    return B200Q_ECUDA;
  }
  const LatentTokens a{qa, (const bf16*)cache, block_table, row_seq, positions, sink, (const bf16*)gate, (bf16*)out, failed,
                       (float)(scale * 1.4426950408889634), bt_stride, heads, R, R + P, shift_of(block_size), window, ld_gate};
#define BY_RANK(MT)                                             \
  do {                                                          \
    if (R == 128) return launch_latent_tokens<MT, 2>(a, T, st); \
    if (R == 256) return launch_latent_tokens<MT, 4>(a, T, st); \
    if (R == 384) return launch_latent_tokens<MT, 6>(a, T, st); \
    return launch_latent_tokens<MT, 8>(a, T, st);               \
  } while (0)
  if (heads > 16) BY_RANK(2);
  BY_RANK(1);
#undef BY_RANK
}

bool portion_attn_gqa_ok(const float* qs, const void* cache, const void* out, int kv_heads, int dim, int vdim, int block_size) {
  return portion_attn_on() && (dim == 64 || dim == 128) && (vdim == 64 || vdim == 128) && shift_of(block_size) >= 0 &&
         ((reinterpret_cast<uintptr_t>(qs) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(out)) & 15) == 0 &&
         kv_heads > 0;
}

int portion_attn_gqa(const float* qs, const void* cache, const int32_t* block_table, int bt_stride, const int32_t* seq_desc,
                     int n_seqs, int longest, int T, int heads, int kv_heads, int dim, int vdim, int block_size, int window,
                     const float* sink, const void* gate, int ld_gate, int channel_gate, void* out, cudaStream_t st) {
  PortionAttn a{};
  a.q32 = qs;
  a.cache = (const bf16*)cache;
  a.block_table = block_table;
  a.seq_desc = seq_desc;
  a.sink = sink;
  a.gate = (const bf16*)gate;
  a.out = (bf16*)out;
  a.qmul = 1.4426950408889634f;
  a.bt_stride = bt_stride;
  a.heads = heads;
  a.kv_heads = kv_heads;
  a.dim = dim;
  a.row = kv_heads * (dim + vdim);
  a.bs_shift = shift_of(block_size);
  a.window = window;
  a.ld_gate = ld_gate;
  a.channel_gate = channel_gate;
  const bool tokens = heads / kv_heads <= 16;  // groups of more heads than a tile has rows: the portions' kernel serves all
  a.skip_single = tokens ? 1 : 0;
#define BY_SIZE(F, ...)                                                              \
  (dim == 64 ? (vdim == 64 ? F<64, 64>(__VA_ARGS__) : F<64, 128>(__VA_ARGS__))       \
             : (vdim == 64 ? F<128, 64>(__VA_ARGS__) : F<128, 128>(__VA_ARGS__)))
  if (T > n_seqs || !tokens) {
    if (int rc = BY_SIZE(launch_gqa_portions, a, n_seqs, longest, st)) return rc;
    if ((long long)n_seqs * longest == T) return B200Q_OK;  // portions of one length: no single tokens
  }
  if (!tokens) return B200Q_OK;
  return BY_SIZE(launch_tokens, a, n_seqs, st);
#undef BY_SIZE
}

}  // namespace b200q

using namespace b200q;

extern "C" {

int b200q_latent_expand_ok(int heads, int dim, int rot_dim, int vdim, int kv_rank, int block_size, int dtype) {
  const int dk = dim + rot_dim;
  return dtype == B200Q_DTYPE_BF16 && portion_attn_on() && heads > 0 && (dk == 64 || dk == 128 || dk == 192) && dim > 0 &&
                 dim % 8 == 0 && (vdim == 64 || vdim == 128) && kv_rank % 64 == 0 && (heads * dim) % 64 == 0 &&
                 shift_of(block_size) >= 0
             ? 1
             : 0;
}

int b200q_latent_gather(const void* cache, const int32_t* block_table, int bt_stride, const int32_t* seq_desc, int n_seqs,
                        int longest_span, int window, int block_size, int kv_rank, int rot_dim, int max_rows, void* out,
                        int32_t* span, void* stream) {
  B200Q_CHECK_ARG(cache && block_table && seq_desc && out && span && n_seqs > 0 && longest_span > 0 && window >= 0 &&
                      kv_rank > 0 && kv_rank % 8 == 0 && rot_dim >= 0 && rot_dim % 8 == 0 && shift_of(block_size) >= 0 &&
                      ((reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(out)) & 15) == 0,
                  "latent_gather: bad argument (kv_rank=%d rot_dim=%d)", kv_rank, rot_dim);
  dim3 grid(n_seqs, (longest_span + 63) / 64);
  B200Q_CHECK_ARG(grid.y <= 65535, "latent_gather: span of %d rows too long", longest_span);
  latent_gather_kernel<<<grid, 256, 0, as_stream(stream)>>>((const bf16*)cache, block_table, bt_stride, seq_desc, window,
                                                            shift_of(block_size), kv_rank, kv_rank + rot_dim, max_rows,
                                                            (bf16*)out, (int2*)span);
  B200Q_LAUNCH_CHECK();
  return B200Q_OK;
}

int b200q_latent_portion_attn(const void* q, int ldq, const float* qa, const void* keys, const void* values, const int32_t* span,
                              const void* cache, const int32_t* block_table, int bt_stride, const int32_t* seq_desc, int n_seqs,
                              int longest, int heads, int dim, int rot_dim, int vdim, int kv_rank, int block_size, int window,
                              float scale, const float* sink, const void* gate, int ld_gate, void* out, void* stream) {
  B200Q_CHECK_ARG(q && qa && keys && values && span && cache && block_table && seq_desc && out && n_seqs > 0 && longest > 0 &&
                      window >= 0 && b200q_latent_expand_ok(heads, dim, rot_dim, vdim, kv_rank, block_size, B200Q_DTYPE_BF16) &&
                      ldq % 8 == 0 && (dim + rot_dim) % 8 == 0 && (!gate || ld_gate >= heads) &&
                      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(qa) | reinterpret_cast<uintptr_t>(keys) |
                        reinterpret_cast<uintptr_t>(values) | reinterpret_cast<uintptr_t>(cache)) & 15) == 0,
                  "latent_portion_attn: bad argument (heads=%d dim=%d rot_dim=%d vdim=%d kv_rank=%d)", heads, dim, rot_dim, vdim,
                  kv_rank);
  PortionAttn a{};
  a.q32 = qa;
  a.q16 = (const bf16*)q;
  a.cache = (const bf16*)cache;
  a.kx = (const bf16*)keys;
  a.vx = (const bf16*)values;
  a.span = (const int2*)span;
  a.block_table = block_table;
  a.seq_desc = seq_desc;
  a.sink = sink;
  a.gate = (const bf16*)gate;
  a.out = (bf16*)out;
  a.qmul = (float)(scale * 1.4426950408889634);
  a.bt_stride = bt_stride;
  a.heads = heads;
  a.kv_heads = heads;
  a.dim = dim;
  a.rot_dim = rot_dim;
  a.kv_rank = kv_rank;
  a.row = kv_rank + rot_dim;
  a.ldq = ldq;
  a.bs_shift = shift_of(block_size);
  a.window = window;
  a.ld_gate = ld_gate;
  a.skip_single = 1;
  cudaStream_t st = as_stream(stream);
  const int dk = dim + rot_dim;
#define PORTIONS(DK) \
  return vdim == 64 ? launch_portions<DK, 64, true>(a, n_seqs, longest, st) : launch_portions<DK, 128, true>(a, n_seqs, longest, st)
  if (dk == 64) PORTIONS(64);
  if (dk == 128) PORTIONS(128);
  PORTIONS(192);
#undef PORTIONS
}

}  // extern "C"
