// Latent attention over a paged cache of latents: one row [c (rp) | r (ep)] per token, shared by all heads.
//
//   latent_rows_kernel     one CTA per token: rms norm of the latent and rotation of the shared key part into the cache row; the
//                          rotated query parts go beside the latent queries (absorbed rows) or, with the unrotated parts, into the
//                          expanded form's padded heads (expanded rows)
//   head_gemm_kernel       out[row, head, :] = W[head] in[row, head, :], mma.sync, 64 rows x 64 columns of one head per CTA: the
//                          absorbed W_uk on the query side and W_uv on the output side
//   latent_attn_kernel     absorbed attention (bf16): 16 or 32 (token, head) rows per CTA against 64-token tiles of the cache, which
//                          serve as keys (full width) and values (first rp columns).  Eight warps: 8 keys each for the scores,
//                          an eighth of the latent each for the output.  Split over the keys where the grid is small
//                          (latent_merge_kernel).  Decode rows and short portions alike.
//   latent_attn_f32_kernel the same in fp32, one warp per (row, head)
//   latent_gather_kernel, latent_pages_kernel   expanded form: visible cache rows as a matrix; its product with [W_uk; W_uv] to
//                          per-head K and V pages in the layout of the attention kernels
#include "common.cuh"
#include "host_api.h"
#include "mma_util.cuh"
#include "tc_util.cuh"
#include "vec_io.cuh"

namespace atlas {

template <typename T>
struct LatentRowParams {
  const T* q; long long ldq;                   // [T, H, rope + nope]
  const float* ckv; long long ldc;             // [T, rank + rope]
  const float* norm_w;
  const int* positions; const float* rope_table;     // [pos, rotary]: cos half, sin half
  const int* slot_mapping; const int* row_map; // row_map: >= 0 absorbed row, < 0 expanded row -(r + 1); null = all absorbed in place
  T* cache;                                    // [slots, rp + ep]
  T* qa;                                       // [absorbed rows, H, rp + ep]: the rotated part is written here
  T* qx;                                       // [expanded rows, H, dx]
  int H, nope, rope, rotary, rank, rp, ep, dx;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(128)
latent_rows_kernel(const LatentRowParams<T> p) {
  __shared__ float red[4];
  chain_trigger();
  chain_wait();
  const int t = blockIdx.x, tid = threadIdx.x, W = p.rp + p.ep, half = p.rotary >> 1;
  const float* cs = p.rope_table + (long long)p.positions[t] * p.rotary;
  auto turned = [&](auto at, int d) -> float { // component d of a rotated part whose component i is at(i)
    if (d >= p.rotary) return at(d);
    return d < half ? at(d) * cs[d] - at(d + half) * cs[half + d] : at(d) * cs[d - half] + at(d - half) * cs[d];
  };
  const int slot = p.slot_mapping[t];
  const float* c = p.ckv + t * p.ldc;
  if (slot >= 0) {
    float ss = 0.f;
    for (int e = tid; e < p.rank; e += 128) ss += c[e] * c[e];
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    const float rstd = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)p.rank + p.eps);
    T* row = p.cache + (long long)slot * W;
    for (int e = tid; e < p.rp; e += 128) row[e] = from_f32<T>(e < p.rank ? c[e] * rstd * p.norm_w[e] : 0.f);
    for (int e = tid; e < p.ep; e += 128)
      row[p.rp + e] = from_f32<T>(e < p.rope ? turned([&](int i) { return c[p.rank + i]; }, e) : 0.f);
  }
  const int dst = p.row_map ? p.row_map[t] : t;
  const T* q = p.q + t * p.ldq;
  const int qd = p.rope + p.nope;
  if (dst >= 0) {
    T* out = p.qa + (long long)dst * p.H * W + p.rp;
    for (int i = tid; i < p.H * p.ep; i += 128) {
      const int h = i / p.ep, e = i % p.ep;
      out[(long long)h * W + e] = from_f32<T>(e < p.rope ? turned([&](int j) { return to_f32(q[h * qd + j]); }, e) : 0.f);
    }
  } else {
    T* out = p.qx + (long long)(-dst - 1) * p.H * p.dx;
    for (int i = tid; i < p.H * p.dx; i += 128) {
      const int h = i / p.dx, e = i % p.dx;
      out[i] = from_f32<T>(e < p.rope ? turned([&](int j) { return to_f32(q[h * qd + j]); }, e) : (e < qd ? to_f32(q[h * qd + e]) : 0.f));
    }
  }
}

// ----------------------------------------------------------------------------- products per head
constexpr int kHgM = 64, kHgN = 64, kHgK = 128, kHgS = kHgK + 8;

struct HeadGemmParams {
  const __nv_bfloat16* in; long long in_row; int in_head;        // element (row, head, k) at in[row * in_row + head * in_head + k]
  const __nv_bfloat16* w;                                        // [H, N, K]
  __nv_bfloat16* out; long long out_row; int out_head;
  const int* in_rows; const int* out_rows;                       // row lists (null = identity)
  int rows, N, K, vec;
};

__global__ void __launch_bounds__(128)
head_gemm_kernel(const HeadGemmParams p) {
  extern __shared__ __align__(16) uint8_t hg_smem[];
  __nv_bfloat16* sa = reinterpret_cast<__nv_bfloat16*>(hg_smem);                  // [2][64][kHgS]
  __nv_bfloat16* sb = sa + 2 * kHgM * kHgS;
  chain_trigger();
  const int head = blockIdx.y, n0 = blockIdx.x * kHgN, m0 = blockIdx.z * kHgM;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int rows = min(kHgM, p.rows - m0), mt = (rows + 15) / 16;
  const __nv_bfloat16* wh = p.w + (long long)head * p.N * p.K;
  auto stage = [&](int buf, int k0, bool weights) {
    const int limit = weights ? p.N - n0 : rows, want = weights ? kHgN : mt * 16;
    __nv_bfloat16* dst = (weights ? sb : sa) + buf * kHgM * kHgS;
    for (int i = tid; i < want * (kHgK / 8); i += 128) {
      const int r = i / (kHgK / 8), c = (i % (kHgK / 8)) * 8;
      const bool live = r < limit && k0 + c < p.K;
      const __nv_bfloat16* src = wh;
      if (live && weights) src = wh + (long long)(n0 + r) * p.K + k0 + c;
      else if (live) src = p.in + (long long)(p.in_rows ? p.in_rows[m0 + r] : m0 + r) * p.in_row + head * p.in_head + k0 + c;
      if (p.vec) {
        cp_async16(smem_u32(dst + r * kHgS + c), src, live);
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) dst[r * kHgS + c + e] = live && k0 + c + e < p.K ? src[e] : __float2bfloat16_rn(0.f);
      }
    }
  };
  const int nk = (p.K + kHgK - 1) / kHgK;
  stage(0, 0, true);                           // weights do not depend on the previous kernel
  chain_wait();
  stage(0, 0, false);
  cp_async_commit();
  float acc[4][2][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
  const int a_row = lane & 15, a_col = (lane >> 4) * 8;
  const int b_row = (lane & 7) + ((lane >> 4) << 3), b_col = ((lane >> 3) & 1) * 8;
  for (int i = 0; i < nk; ++i) {
    if (i + 1 < nk) { stage((i + 1) & 1, (i + 1) * kHgK, true); stage((i + 1) & 1, (i + 1) * kHgK, false); }
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t ua = smem_u32(sa + (i & 1) * kHgM * kHgS), ub = smem_u32(sb + (i & 1) * kHgM * kHgS);
#pragma unroll
    for (int kk = 0; kk < kHgK / 16; ++kk) {
      uint32_t bb[4];
      ldsm4(ub + ((warp * 16 + b_row) * kHgS + kk * 16 + b_col) * 2, bb);
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        if (m >= mt) break;
        uint32_t a[4];
        ldsm4(ua + ((m * 16 + a_row) * kHgS + kk * 16 + a_col) * 2, a);
        mma16816(acc[m][0], a, bb[0], bb[1]);
        mma16816(acc[m][1], a, bb[2], bb[3]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int r = m * 16 + g + 8 * hh;
      if (r >= rows) continue;
      __nv_bfloat16* orow = p.out + (long long)(p.out_rows ? p.out_rows[m0 + r] : m0 + r) * p.out_row + head * p.out_head;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int n = n0 + warp * 16 + j * 8 + 2 * t4 + e;
          if (n < p.N) orow[n] = __float2bfloat16_rn(acc[m][j][2 * hh + e]);
        }
    }
}

// ----------------------------------------------------------------------------- absorbed attention
constexpr int kLtTok = 64, kLtWarps = 8, kLtPS = kLtTok + 8;

template <typename T>
struct LatentAttnParams {
  const T* q;                                  // [rows, H, W]
  const T* cache;                              // [blocks, bs, W]
  T* out;                                      // [rows, H, rp]
  float* part_o; float* part_ml;               // [rows * H, splits, rp], [rows * H, splits, 2]
  const int* block_tables; int bt_ld;
  const int* seq_lens; const int* query_start_loc;
  const int* row_start;                        // [B] first row of a sequence in q / out (null = query_start_loc)
  const int* tile_seq; const int* tile_r0;     // (sequence, first flattened (token, head) row); null: tile z of sequence blockIdx.x
  int H, rp, ep, block_size, window, splits, stages;
  float scale;
};

template <int NT, int MT>
__global__ void __launch_bounds__(32 * kLtWarps)
latent_attn_kernel(const LatentAttnParams<__nv_bfloat16> p) {
  constexpr int M = 16 * MT;
  extern __shared__ __align__(16) uint8_t lt_smem[];
  const int W = p.rp + p.ep, WS = W + 8;
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(lt_smem);                 // [M][WS]
  __nv_bfloat16* sp = sq + M * WS;                                               // [M][kLtPS]
  float* smax = reinterpret_cast<float*>(sp + M * kLtPS);                        // [8][M]
  float* ssum = smax + kLtWarps * M;
  __nv_bfloat16* skv = reinterpret_cast<__nv_bfloat16*>(ssum + kLtWarps * M);    // [stages][64][WS]
  chain_trigger();
  chain_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int b = p.tile_seq ? p.tile_seq[blockIdx.x] : blockIdx.x;
  const int r0 = p.tile_seq ? p.tile_r0[blockIdx.x] : blockIdx.z * M, split = blockIdx.y;
  const int q0 = p.query_start_loc[b], q_len = p.query_start_loc[b + 1] - q0, L = p.seq_lens[b], ctx = L - q_len;
  const int n_flat = q_len * p.H;              // (token, head) rows of the sequence
  const int row0 = p.row_start ? p.row_start[b] : q0;
  const long long flat0 = (long long)row0 * p.H + r0;
  if (r0 >= n_flat) return;
  auto low = [&](int pos) { return p.window > 0 ? max(0, pos - p.window + 1) : 0; };
  const int last = min(r0 + M, n_flat) - 1;
  const int key_lo = low(ctx + r0 / p.H), key_hi = ctx + last / p.H + 1;         // keys some row of the tile sees
  const int tiles = (key_hi - key_lo + kLtTok - 1) / kLtTok, per = (tiles + p.splits - 1) / p.splits;
  const int j0 = split * per, j1 = min(tiles, j0 + per);
  const int* bt = p.block_tables + (long long)b * p.bt_ld;

  // queries of the tile (zeros past the end)
  const int CW = W / 8;
  for (int i = tid; i < M * CW; i += 32 * kLtWarps) {
    const int r = i / CW, c = (i % CW) * 8;
    cp_async16(smem_u32(sq + r * WS + c), p.q + (flat0 + (r0 + r < n_flat ? r : 0)) * W + c, r0 + r < n_flat);
  }
  auto fetch = [&](int j, int st) {
    const int k0 = key_lo + j * kLtTok;
    for (int i = tid; i < kLtTok * CW; i += 32 * kLtWarps) {
      const int r = i / CW, c = (i % CW) * 8, key = k0 + r;
      const bool live = key < key_hi;
      const long long row = live ? (long long)bt[key / p.block_size] * p.block_size + key % p.block_size : 0;
      cp_async16(smem_u32(skv + ((long long)st * kLtTok + r) * WS + c), p.cache + row * W + c, live);
    }
  };
  int pos[MT][2], lo[MT][2];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = r0 + m * 16 + g + 8 * h;
      pos[m][h] = r < n_flat ? ctx + r / p.H : -1;
      lo[m][h] = low(pos[m][h]);
    }
  float o[MT][NT][4], mr[MT][2], lr[MT][2];
#pragma unroll
  for (int m = 0; m < MT; ++m) {
    mr[m][0] = mr[m][1] = -INFINITY;
    lr[m][0] = lr[m][1] = 0.f;
#pragma unroll
    for (int j = 0; j < NT; ++j) o[m][j][0] = o[m][j][1] = o[m][j][2] = o[m][j][3] = 0.f;
  }
  const float sl2 = p.scale * 1.4426950408889634f;
  const int a_row = lane & 15, a_col = (lane >> 4) * 8;
  const uint32_t uq = smem_u32(sq), up = smem_u32(sp);
  const int d0 = warp * NT * 8;                // this warp's latent columns

  if (j0 < j1) fetch(j0, 0);
  cp_async_commit();
  for (int j = j0; j < j1; ++j) {
    const int st = p.stages == 2 ? (j - j0) & 1 : 0;
    if (p.stages == 2 && j + 1 < j1) fetch(j + 1, st ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t ukv = smem_u32(skv + (long long)st * kLtTok * WS);
    // ---- scores of keys 8 warp .. 8 warp + 7
    float s[MT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m) s[m][0] = s[m][1] = s[m][2] = s[m][3] = 0.f;
    {
      // two k-steps per ldmatrix.x4: matrices are the key rows' columns 0..7, 8..15, 16..23, 24..31
      const uint32_t bk = ukv + ((warp * 8 + (lane & 7)) * WS + (lane >> 3) * 8) * 2;
      int kk = 0;
      for (; kk + 32 <= W; kk += 32) {
        uint32_t bb[4];
        ldsm4(bk + kk * 2, bb);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t a[4];
          ldsm4(uq + ((m * 16 + a_row) * WS + kk + a_col) * 2, a);
          mma16816(s[m], a, bb[0], bb[1]);
          ldsm4(uq + ((m * 16 + a_row) * WS + kk + 16 + a_col) * 2, a);
          mma16816(s[m], a, bb[2], bb[3]);
        }
      }
      if (kk < W) {
        uint32_t b0, b1;
        ldsm2(ukv + ((warp * 8 + (lane & 7)) * WS + kk + ((lane >> 3) & 1) * 8) * 2, b0, b1);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t a[4];
          ldsm4(uq + ((m * 16 + a_row) * WS + kk + a_col) * 2, a);
          mma16816(s[m], a, b0, b1);
        }
      }
    }
    const int key = key_lo + j * kLtTok + warp * 8 + 2 * t4;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float& x = s[m][2 * h + e];
          x = key + e <= pos[m][h] && key + e >= lo[m][h] ? x * sl2 : -INFINITY;
        }
        float mx = fmaxf(s[m][2 * h], s[m][2 * h + 1]);
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        if (t4 == 0) smax[warp * M + m * 16 + g + 8 * h] = mx;
      }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = m * 16 + g + 8 * h;
        float mx = mr[m][h];
#pragma unroll
        for (int w = 0; w < kLtWarps; ++w) mx = fmaxf(mx, smax[w * M + r]);
        const float ref = mx == -INFINITY ? 0.f : mx, alpha = exp2f(mr[m][h] - ref);        // nothing seen yet: 0
        const float p0 = exp2f(s[m][2 * h] - ref), p1 = exp2f(s[m][2 * h + 1] - ref);
        lr[m][h] = lr[m][h] * alpha + p0 + p1;
        mr[m][h] = mx;
        *reinterpret_cast<uint32_t*>(sp + r * kLtPS + warp * 8 + 2 * t4) = pack_bf16x2(p0, p1);
#pragma unroll
        for (int n = 0; n < NT; ++n) { o[m][n][2 * h] *= alpha; o[m][n][2 * h + 1] *= alpha; }
      }
    __syncthreads();
    // ---- output: this warp's columns over all 64 keys
    if (d0 < p.rp) {
#pragma unroll
      for (int kk = 0; kk < kLtTok / 16; ++kk) {
        uint32_t a[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) ldsm4(up + ((m * 16 + a_row) * kLtPS + kk * 16 + a_col) * 2, a[m]);
        if constexpr (NT == 1) {
          uint32_t b0, b1;                     // one n8 tile: matrices keys 0..7 and 8..15
          asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];\n"
                       : "=r"(b0), "=r"(b1) : "r"(ukv + ((kk * 16 + a_row) * WS + d0) * 2) : "memory");
#pragma unroll
          for (int m = 0; m < MT; ++m) mma16816(o[m][0], a[m], b0, b1);
        } else {
#pragma unroll
          for (int n = 0; n < NT / 2; ++n) {
            if (d0 + n * 16 >= p.rp) break;
            uint32_t x[4];
            ldsm4t(ukv + ((kk * 16 + a_row) * WS + d0 + n * 16 + a_col) * 2, x);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              mma16816(o[m][2 * n], a[m], x[0], x[1]);
              mma16816(o[m][2 * n + 1], a[m], x[2], x[3]);
            }
          }
        }
      }
    }
    __syncthreads();                           // the tile's buffers are free
    if (p.stages == 1 && j + 1 < j1) {
      fetch(j + 1, 0);
      cp_async_commit();
    }
  }
  cp_async_wait<0>();
  // ---- sums over the warps' keys, output
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float l = lr[m][h];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      if (t4 == 0) ssum[warp * M + m * 16 + g + 8 * h] = l;
    }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = m * 16 + g + 8 * h;
      if (r0 + r >= n_flat) continue;
      float l = 0.f;
#pragma unroll
      for (int w = 0; w < kLtWarps; ++w) l += ssum[w * M + r];
      const long long flat = flat0 + r;
      if (p.splits == 1) {
        const float inv = 1.f / l;             // a row sees at least itself
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const int d = d0 + n * 8 + 2 * t4;
          if (d < p.rp) *reinterpret_cast<uint32_t*>(p.out + flat * p.rp + d) = pack_bf16x2(o[m][n][2 * h] * inv, o[m][n][2 * h + 1] * inv);
        }
      } else {
        float* po = p.part_o + (flat * p.splits + split) * p.rp;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const int d = d0 + n * 8 + 2 * t4;
          if (d < p.rp) *reinterpret_cast<float2*>(po + d) = make_float2(o[m][n][2 * h], o[m][n][2 * h + 1]);
        }
        if (warp == 0 && t4 == 0) {
          p.part_ml[(flat * p.splits + split) * 2] = mr[m][h];
          p.part_ml[(flat * p.splits + split) * 2 + 1] = l;
        }
      }
    }
}

// one CTA per (token, head) row
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, __nv_bfloat16* out, int rp, int splits) {
  chain_trigger();
  chain_wait();
  const long long flat = blockIdx.x;
  float m = -INFINITY, l = 0.f;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, part_ml[(flat * splits + s) * 2]);
  for (int s = 0; s < splits; ++s) {
    const float ms = part_ml[(flat * splits + s) * 2];
    l += ms == -INFINITY ? 0.f : exp2f(ms - m) * part_ml[(flat * splits + s) * 2 + 1];
  }
  const float inv = 1.f / l;
  for (int d = threadIdx.x * 2; d < rp; d += 256) {
    float a0 = 0.f, a1 = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float ms = part_ml[(flat * splits + s) * 2];
      if (ms == -INFINITY) continue;           // the split saw no key of this row
      const float f = exp2f(ms - m);
      const float2 v = *reinterpret_cast<const float2*>(part_o + (flat * splits + s) * rp + d);
      a0 += f * v.x;
      a1 += f * v.y;
    }
    *reinterpret_cast<uint32_t*>(out + flat * rp + d) = pack_bf16x2(a0 * inv, a1 * inv);
  }
}

constexpr int kLfMax = 32;                     // latent components per lane: ranks up to 1024
__global__ void __launch_bounds__(128)
latent_attn_f32_kernel(const LatentAttnParams<float> p, int B, int T) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, W = p.rp + p.ep;
  const long long unit = (long long)blockIdx.x * 4 + warp;
  if (unit >= (long long)T * p.H) return;
  const int t = (int)(unit / p.H);
  int lo_b = 0, hi_b = B;                      // the sequence that owns row t
  while (lo_b + 1 < hi_b) {
    const int mid = (lo_b + hi_b) >> 1;
    if (p.query_start_loc[mid] <= t) lo_b = mid; else hi_b = mid;
  }
  const int pos = p.seq_lens[lo_b] - (p.query_start_loc[lo_b + 1] - t);
  if (pos < 0) return;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int* bt = p.block_tables + (long long)lo_b * p.bt_ld;
  const float* q = p.q + unit * W;
  float o[kLfMax], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int i = 0; i < kLfMax; ++i) o[i] = 0.f;
  for (int j0 = lo; j0 <= pos; j0 += 32) {
    const int j = j0 + lane;
    const bool ok = j <= pos;
    float s = -INFINITY;
    if (ok) {
      const float4* kr = reinterpret_cast<const float4*>(p.cache + ((long long)bt[j / p.block_size] * p.block_size + j % p.block_size) * W);
      s = 0.f;
      for (int d = 0; d < W / 4; ++d) {
        const float4 kv = __ldg(kr + d), qv = __ldg(reinterpret_cast<const float4*>(q) + d);
        s += kv.x * qv.x + kv.y * qv.y + kv.z * qv.z + kv.w * qv.w;
      }
      s *= p.scale;
    }
    const float top = fmaxf(m, warp_max(s));
    const float f = m == -INFINITY ? 0.f : expf(m - top), e = ok ? expf(s - top) : 0.f;
    l = l * f + warp_sum(e);
    m = top;
#pragma unroll
    for (int i = 0; i < kLfMax; ++i) o[i] *= f;
    const int n = min(32, pos - j0 + 1);
    for (int jj = 0; jj < n; ++jj) {
      const float w = __shfl_sync(0xffffffffu, e, jj);
      const int key = j0 + jj;
      const float* row = p.cache + ((long long)bt[key / p.block_size] * p.block_size + key % p.block_size) * W;
#pragma unroll
      for (int i = 0; i < kLfMax; ++i)
        if (i * 32 + lane < p.rp) o[i] = fmaf(w, __ldg(row + i * 32 + lane), o[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < kLfMax; ++i)
    if (i * 32 + lane < p.rp) p.out[unit * p.rp + i * 32 + lane] = o[i] / l;
}

// ----------------------------------------------------------------------------- expanded form
// page i of the scratch pages: 16 tokens from token 16 page_idx[i] of sequence page_seq[i]; out [pages * 16, rp], zeros past the end
__global__ void __launch_bounds__(128)
latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_tables, int bt_ld, const int* __restrict__ seq_lens,
                     const int* __restrict__ page_seq, const int* __restrict__ page_idx, int block_size, int rp, int W, __nv_bfloat16* out) {
  const int i = blockIdx.x, b = page_seq[i], t0 = page_idx[i] * 16, L = seq_lens[b];
  const int C = rp / 8;
  const long long base = (long long)block_tables[(long long)b * bt_ld + t0 / block_size] * block_size + t0 % block_size;
  for (int e = threadIdx.x; e < 16 * C; e += 128) {
    const int r = e / C, c = (e % C) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (t0 + r < L) v = *reinterpret_cast<const uint4*>(cache + (base + r) * W + c);
    *reinterpret_cast<uint4*>(out + ((long long)i * 16 + r) * rp + c) = v;
  }
}

// kv [pages * 16, H * (nope + vd)] (per head: unrotated key, value) and the cache's rotated parts -> K pages [page, H, 16, dx] with
// rows [rope | nope | 0], V pages [page, H, dx, 16]
__global__ void __launch_bounds__(128)
latent_pages_kernel(const __nv_bfloat16* __restrict__ kv, const __nv_bfloat16* __restrict__ cache, const int* __restrict__ block_tables,
                    int bt_ld, const int* __restrict__ seq_lens, const int* __restrict__ page_seq, const int* __restrict__ page_idx,
                    int block_size, int H, int nope, int rope, int vd, int rp, int W, int dx, __nv_bfloat16* kp, __nv_bfloat16* vp) {
  extern __shared__ __nv_bfloat16 lp_smem[];   // [16][vd + 2]
  const int i = blockIdx.x, h = blockIdx.y, b = page_seq[i], t0 = page_idx[i] * 16, L = seq_lens[b], tid = threadIdx.x;
  const long long base = (long long)block_tables[(long long)b * bt_ld + t0 / block_size] * block_size + t0 % block_size;
  const __nv_bfloat16* src = kv + (long long)i * 16 * H * (nope + vd) + h * (nope + vd);
  const long long row = (long long)H * (nope + vd);
  const __nv_bfloat16 zero = __float2bfloat16_rn(0.f);
  __nv_bfloat16* kd = kp + ((long long)i * H + h) * 16 * dx;
  if (nope % 2 == 0 && rope % 2 == 0 && vd % 2 == 0) {           // pairs
    for (int e = tid; e < 16 * dx / 2; e += 128) {
      const int r = e / (dx / 2), c = (e % (dx / 2)) * 2;
      uint32_t v = 0u;
      if (t0 + r < L) {
        if (c < rope) v = *reinterpret_cast<const uint32_t*>(cache + (base + r) * W + rp + c);
        else if (c < rope + nope) v = *reinterpret_cast<const uint32_t*>(src + r * row + c - rope);
      }
      *reinterpret_cast<uint32_t*>(kd + r * dx + c) = v;
    }
    for (int e = tid; e < 16 * vd / 2; e += 128) {
      const int r = e / (vd / 2), c = (e % (vd / 2)) * 2;
      *reinterpret_cast<uint32_t*>(lp_smem + r * (vd + 2) + c) = *reinterpret_cast<const uint32_t*>(src + r * row + nope + c);
    }
  } else {
    for (int e = tid; e < 16 * dx; e += 128) {
      const int r = e / dx, c = e % dx;
      __nv_bfloat16 v = zero;
      if (t0 + r < L) {
        if (c < rope) v = cache[(base + r) * W + rp + c];
        else if (c < rope + nope) v = src[r * row + c - rope];
      }
      kd[e] = v;
    }
    for (int e = tid; e < 16 * vd; e += 128) {
      const int r = e / vd, c = e % vd;
      lp_smem[r * (vd + 2) + c] = src[r * row + nope + c];
    }
  }
  __syncthreads();
  __nv_bfloat16* vdst = vp + ((long long)i * H + h) * 16 * dx;
  for (int e = tid; e < dx * 2; e += 128) {    // eight tokens of one value channel
    const int d = e >> 1, r8 = (e & 1) * 8;
    __nv_bfloat16 x[8];
#pragma unroll
    for (int r = 0; r < 8; ++r) x[r] = d < vd && t0 + r8 + r < L ? lp_smem[(r8 + r) * (vd + 2) + d] : zero;
    *reinterpret_cast<uint4*>(vdst + d * 16 + r8) = *reinterpret_cast<const uint4*>(x);
  }
}

// out[rows[i], h, 0..vd) = in[i, h, 0..vd) of padded heads (width dx)
__global__ void __launch_bounds__(256)
latent_unpad_kernel(const __nv_bfloat16* __restrict__ in, const int* __restrict__ rows, int H, int vd, int dx, __nv_bfloat16* out) {
  const long long i = blockIdx.x, dst = rows ? rows[i] : i;
  if (vd % 8 == 0) {
    for (int e = threadIdx.x; e < H * vd / 8; e += 256) {
      const int h = e / (vd / 8), d = (e % (vd / 8)) * 8;
      *reinterpret_cast<uint4*>(out + dst * H * vd + h * vd + d) = *reinterpret_cast<const uint4*>(in + (i * H + h) * dx + d);
    }
  } else {
    for (int e = threadIdx.x; e < H * vd; e += 256) out[dst * H * vd + e] = in[(i * H + e / vd) * dx + e % vd];
  }
}

template <typename T>
static int latent_rows(const void* q, long long ldq, const float* ckv, long long ldc, const float* norm_w, const int* positions, const float* rope,
                       const int* slot_mapping, const int* row_map, void* cache, void* qa, void* qx, int rows, int H, int nope, int rope_dim,
                       int rotary, int rank, int rp, int ep, int dx, float eps, cudaStream_t st) {
  LatentRowParams<T> p = {reinterpret_cast<const T*>(q), ldq, ckv, ldc, norm_w, positions, rope, slot_mapping, row_map, reinterpret_cast<T*>(cache),
                          reinterpret_cast<T*>(qa), reinterpret_cast<T*>(qx), H, nope, rope_dim, rotary, rank, rp, ep, dx, eps};
  launch_chain_if(rows <= 256, latent_rows_kernel<T>, dim3(rows), dim3(128), 0, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <int NT, int MT>
static int launch_latent(LatentAttnParams<__nv_bfloat16>& p, dim3 grid, cudaStream_t st) {
  constexpr int M = 16 * MT;
  const int WS = p.rp + p.ep + 8, fixed = M * WS * 2 + M * kLtPS * 2 + 2 * kLtWarps * M * 4, stage = kLtTok * WS * 2;
  p.stages = fixed + 2 * stage <= 220 * 1024 ? 2 : 1;
  const int smem = fixed + p.stages * stage;
  if (smem > 226 * 1024) return -3;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(latent_attn_kernel<NT, MT>), smem) != cudaSuccess) return -20;
  return launch_chain(latent_attn_kernel<NT, MT>, grid, dim3(32 * kLtWarps), (size_t)smem, st, p) == cudaSuccess ? 0 : -21;
}
template <int MT>
static int launch_latent_nt(LatentAttnParams<__nv_bfloat16>& p, dim3 grid, cudaStream_t st) {
  if (p.rp <= 64) return launch_latent<1, MT>(p, grid, st);
  if (p.rp <= 128) return launch_latent<2, MT>(p, grid, st);
  if (p.rp <= 256) return launch_latent<4, MT>(p, grid, st);
  if (p.rp <= 512) return launch_latent<8, MT>(p, grid, st);
  return launch_latent<16, MT>(p, grid, st);
}

}  // namespace atlas

using namespace atlas;
using bf16 = __nv_bfloat16;

// cache [slots, rp + ep] of the activations' dtype; qa [absorbed rows, H, rp + ep], qx [expanded rows, H, dx] (may be null)
extern "C" int atlas_latent_rows(const void* q, long long ldq, const float* ckv, long long ldc, const float* norm_w, const int* positions,
                                 const float* rope, const int* slot_mapping, const int* row_map, void* cache, void* qa, void* qx, int rows,
                                 int H, int nope, int rope_dim, int rotary, int rank, int rp, int ep, int dx, float eps, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (rotary > rope_dim || rotary % 2 || rank > rp || rope_dim > ep || (qx && dx < nope + rope_dim)) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? latent_rows<float>(q, ldq, ckv, ldc, norm_w, positions, rope, slot_mapping, row_map, cache, qa, qx, rows, H, nope, rope_dim, rotary,
                                  rank, rp, ep, dx, eps, st)
             : latent_rows<bf16>(q, ldq, ckv, ldc, norm_w, positions, rope, slot_mapping, row_map, cache, qa, qx, rows, H, nope, rope_dim, rotary,
                                 rank, rp, ep, dx, eps, st);
}

// out[row, head, n] = sum_k w[head, n, k] in[row, head, k] (bf16); row lists may be null
extern "C" int atlas_head_gemm(const void* in, long long in_row, int in_head, const void* w, void* out, long long out_row, int out_head,
                               const int* in_rows, const int* out_rows, int rows, int H, int N, int K, void* stream) {
  if (rows <= 0 || H <= 0) return 0;
  if (N < 1 || K < 1) return -1;
  const bool vec = K % 8 == 0 && in_row % 8 == 0 && in_head % 8 == 0 && ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(w)) & 15) == 0;
  HeadGemmParams p = {reinterpret_cast<const bf16*>(in), in_row, in_head, reinterpret_cast<const bf16*>(w), reinterpret_cast<bf16*>(out), out_row,
                      out_head, in_rows, out_rows, rows, N, K, vec ? 1 : 0};
  constexpr int smem = 4 * kHgM * kHgS * 2;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(head_gemm_kernel), smem) != cudaSuccess) return -20;
  return launch_chain_if(rows <= 256, head_gemm_kernel, dim3((N + kHgN - 1) / kHgN, H, (rows + kHgM - 1) / kHgM), dim3(128), (size_t)smem,
                         reinterpret_cast<cudaStream_t>(stream), p) == cudaSuccess ? 0 : -21;
}

// Absorbed attention.  `tiles` > 0: (tile_seq, tile_r0) list of tiles of 16 * mt flattened (token, head) rows; otherwise every one
// of the B sequences has one query row.  With splits > 1: part_o [rows * H, splits, rp], part_ml [rows * H, splits, 2], rows = the
// rows of q.
extern "C" int atlas_latent_attn(const void* q, const void* cache, void* out, float* part_o, float* part_ml, const int* block_tables,
                                 int bt_ld, const int* seq_lens, const int* query_start_loc, const int* row_start, const int* tile_seq,
                                 const int* tile_r0, int tiles, int B, int rows, int H, int rp, int ep, int block_size, int window, int splits,
                                 int mt, float scale, void* stream) {
  if (B <= 0 || rows <= 0) return 0;
  if (rp % 16 || ep % 16 || rp > 1024 || (mt != 1 && mt != 2) || block_size < 1) return -1;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15) return -2;
  if (splits > 1 && (!part_o || !part_ml)) return -4;
  LatentAttnParams<bf16> p = {reinterpret_cast<const bf16*>(q), reinterpret_cast<const bf16*>(cache), reinterpret_cast<bf16*>(out), part_o, part_ml,
                              block_tables, bt_ld, seq_lens, query_start_loc, row_start, tiles > 0 ? tile_seq : nullptr, tile_r0, H, rp, ep,
                              block_size, window, splits < 1 ? 1 : splits, 1, scale};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(tiles > 0 ? tiles : B, p.splits, tiles > 0 ? 1 : (H + 16 * mt - 1) / (16 * mt));
  const int rc = mt == 1 ? launch_latent_nt<1>(p, grid, st) : launch_latent_nt<2>(p, grid, st);
  if (rc) return rc;
  if (p.splits > 1 &&
      launch_chain(latent_merge_kernel, dim3((unsigned)(rows * H)), dim3(128), 0, st, (const float*)part_o, (const float*)part_ml, p.out, rp, p.splits) != cudaSuccess)
    return -22;
  return 0;
}

// fp32: rows of all sequences of the step
extern "C" int atlas_latent_attn_f32(const float* q, const float* cache, float* out, const int* block_tables, int bt_ld, const int* seq_lens,
                                     const int* query_start_loc, int B, int T, int H, int rp, int ep, int block_size, int window, float scale,
                                     void* stream) {
  if (B <= 0 || T <= 0) return 0;
  if (rp % 4 || ep % 4 || rp > 32 * kLfMax || block_size < 1) return -1;
  LatentAttnParams<float> p = {q, cache, out, nullptr, nullptr, block_tables, bt_ld, seq_lens, query_start_loc, nullptr, nullptr, nullptr, H, rp, ep,
                               block_size, window, 1, 1, scale};
  latent_attn_f32_kernel<<<(unsigned)(((long long)T * H + 3) / 4), 128, 0, reinterpret_cast<cudaStream_t>(stream)>>>(p, B, T);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

extern "C" int atlas_latent_gather(const void* cache, const int* block_tables, int bt_ld, const int* seq_lens, const int* page_seq,
                                   const int* page_idx, int pages, int block_size, int rp, int W, void* out, void* stream) {
  if (pages <= 0) return 0;
  if (rp % 8 || W % 8 || block_size % 16) return -1;
  latent_gather_kernel<<<pages, 128, 0, reinterpret_cast<cudaStream_t>(stream)>>>(reinterpret_cast<const bf16*>(cache), block_tables, bt_ld, seq_lens,
                                                                                 page_seq, page_idx, block_size, rp, W, reinterpret_cast<bf16*>(out));
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

extern "C" int atlas_latent_pages(const void* kv, const void* cache, const int* block_tables, int bt_ld, const int* seq_lens, const int* page_seq,
                                  const int* page_idx, int pages, int block_size, int H, int nope, int rope, int vd, int rp, int W, int dx,
                                  void* k_pages, void* v_pages, void* stream) {
  if (pages <= 0) return 0;
  if (block_size % 16 || dx % 8 || dx < nope + rope || dx < vd || H > 65535) return -1;
  latent_pages_kernel<<<dim3(pages, H), 128, 16 * (vd + 2) * 2, reinterpret_cast<cudaStream_t>(stream)>>>(
      reinterpret_cast<const bf16*>(kv), reinterpret_cast<const bf16*>(cache), block_tables, bt_ld, seq_lens, page_seq, page_idx, block_size, H, nope,
      rope, vd, rp, W, dx, reinterpret_cast<bf16*>(k_pages), reinterpret_cast<bf16*>(v_pages));
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

extern "C" int atlas_latent_unpad(const void* in, const int* rows, int n, int H, int vd, int dx, void* out, void* stream) {
  if (n <= 0) return 0;
  latent_unpad_kernel<<<n, 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(reinterpret_cast<const bf16*>(in), rows, H, vd, dx, reinterpret_cast<bf16*>(out));
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}
