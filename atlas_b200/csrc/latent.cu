// Latent attention over a paged cache of latents: one row [c (rp) | r (ep)] per token, shared by all heads.
//
//   latent_rows_kernel     one CTA per token: rms norm of the latent and rotation of the shared key part into the cache row; the
//                          rotated query parts go beside the latent queries (absorbed rows) or, with the unrotated parts, into the
//                          expanded form's padded heads (expanded rows)
//   head_gemm_kernel       out[row, head, :] = W[head] in[row, head, :], mma.sync, 64 rows x 64 columns of one head per CTA: the
//                          absorbed W_uk on the query side and W_uv on the output side
//   latent_attn_kernel     absorbed attention (bf16): 16 or 32 (token, head) rows per CTA against tiles of the cache, which serve
//                          as keys (full width) and values (first rp columns).  Split over the keys where the grid is small
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
constexpr int kLtKG = 4, kLtMaxStages = 6;     // groups of warps that share a row's width

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
  int H, rp, ep, block_size, bs_shift, window, splits, stages;   // bs_shift: log2 of the block size, -1 if it is none
  float scale;
};

// A tile of TOK keys goes through three steps, each one tile behind the other, with one barrier per tile:
//   scores    warp (kg, tg): k-steps of group kg for the HK keys of part tg -> partial sums in shared memory (with sixteen warps
//             and 32 rows: warp (kg, tg, wm), one 16-row unit each)
//   softmax   TPR threads per row add the kLtKG partial sums, keep the row's maximum and sum, write the probabilities (bf16)
//   output    every warp its NT * 8 columns of the latent over the tile's keys
// so between two barriers the warps work on the scores of tile p + 1, the softmax of tile p and the output of tile p - 1.  Tiles
// arrive through a ring of `stages` (>= 4) buffers.
// KPG: k-steps per warp (HK = 8: taken in pairs), MT: 16-row units
template <int KPG, int NT, int MT, int WARPS, int TOK>
__global__ void __launch_bounds__(32 * WARPS)
latent_attn_kernel(const LatentAttnParams<__nv_bfloat16> p) {
  constexpr int M = 16 * MT, THREADS = 32 * WARPS, TPR = THREADS / M, KPT = TOK / TPR;
  constexpr int WM = MT == 2 && WARPS == 16 ? 2 : 1, MS = MT / WM;               // parts of the rows, 16-row units of a warp's scores
  constexpr int TG = WARPS / kLtKG / WM, HK = TOK / TG, RPW = TOK / WARPS;
  constexpr int PS = TOK + 8, SS = TOK + 4;    // padded rows of the probabilities and of the partial sums
  static_assert(HK == 8 || HK == 16, "eight or sixteen keys per warp");
  static_assert(HK == 16 || KPG % 2 == 0, "pairs of k-steps");
  extern __shared__ __align__(16) uint8_t lt_smem[];
  const int W = p.rp + p.ep, WS = W + 8, CW = W / 8;
  float* spart = reinterpret_cast<float*>(lt_smem);                              // [2][kLtKG][M][SS]
  __nv_bfloat16* sp = reinterpret_cast<__nv_bfloat16*>(spart + 2 * kLtKG * M * SS);        // [2][M][PS]
  float* salpha = reinterpret_cast<float*>(sp + 2 * M * PS);                     // [2][M]
  float* ssum = salpha + 2 * M;                                                  // [M]
  __nv_bfloat16* skv = reinterpret_cast<__nv_bfloat16*>(ssum + M);               // [stages][TOK][WS]
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
  const int tiles = (key_hi - key_lo + TOK - 1) / TOK, per = (tiles + p.splits - 1) / p.splits;
  const int j0 = split * per, n_tiles = max(0, min(tiles, j0 + per) - j0), kv0 = key_lo + j0 * TOK;
  const int* bt = p.block_tables + (long long)b * p.bt_ld;
  const int S = p.stages;

  // A warp copies rows warp, warp + WARPS, .. of a tile; lane i looks up the i-th of them.  The page number is fetched one tile
  // before it is used: nothing waits for it.
  auto page_of = [&](int t) -> int {
    const int key = kv0 + t * TOK + warp + WARPS * (lane & (RPW - 1));
    return t < n_tiles && key < key_hi ? bt[p.bs_shift >= 0 ? key >> p.bs_shift : key / p.block_size] : -1;
  };
  auto fetch = [&](int st, int t, int page) {
    const int key = kv0 + t * TOK + warp + WARPS * (lane & (RPW - 1));
    const int rows = page < 0 ? -1 : page * p.block_size + (p.bs_shift >= 0 ? key & (p.block_size - 1) : key % p.block_size);
    const uint32_t dst = smem_u32(skv + (long long)st * TOK * WS);
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
      const int row = __shfl_sync(0xffffffffu, rows, i);
      const __nv_bfloat16* src = p.cache + (long long)max(row, 0) * W;
#pragma unroll
      for (int u = 0; u < (KPG * kLtKG * 2 + 31) / 32; ++u) {
        const int c = u * 32 + lane;
        if (c < CW) cp_async16(dst + ((warp + WARPS * i) * WS + c * 8) * 2, src + c * 8, row >= 0);
      }
    }
  };
  for (int t = 0; t < S - 2; ++t) {            // one group per tile, empty past the end
    if (t < n_tiles) fetch(t, t, page_of(t));
    cp_async_commit();
  }
  int next = page_of(S - 2);

  // query fragments of this warp's k-steps stay in registers (zero past the row's width)
  const int kg = warp % kLtKG, tg = warp / kLtKG % TG, m0 = warp / (kLtKG * TG) * MS, nks = W / 16;
  auto kstep = [&](int i) { return HK == 8 ? 2 * (kg + kLtKG * (i >> 1)) + (i & 1) : kg + kLtKG * i; };
  uint32_t qf[MS][KPG][4];
#pragma unroll
  for (int m = 0; m < MS; ++m)
#pragma unroll
    for (int i = 0; i < KPG; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = (m0 + m) * 16 + g + 8 * (e & 1), k = kstep(i) * 16 + 2 * t4 + 8 * (e >> 1);
        qf[m][i][e] = r0 + r < n_flat && k < W ? *reinterpret_cast<const uint32_t*>(p.q + (flat0 + r) * W + k) : 0u;
      }
  // softmax: this thread's row and keys
  const int srow = tid / TPR, sc = (tid % TPR) * KPT;
  const int pos = r0 + srow < n_flat ? ctx + (r0 + srow) / p.H : -1, lo = low(pos);
  const float sl2 = p.scale * 1.4426950408889634f;
  float mrun = -INFINITY, lrun = 0.f;
  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < NT; ++j) o[m][j][0] = o[m][j][1] = o[m][j][2] = o[m][j][3] = 0.f;
  const int a_row = lane & 15, a_col = (lane >> 4) * 8;
  const uint32_t ukv0 = smem_u32(skv), up0 = smem_u32(sp), stage_bytes = TOK * WS * 2;
  const int d0 = warp * NT * 8;                // this warp's latent columns

  // ldmatrix addresses inside a tile: this warp's keys at its k-steps (clamped into the row), its latent columns (likewise)
  constexpr int KO = HK == 16 ? KPG : KPG / 2, VO = NT == 1 ? 1 : NT / 2;
  uint32_t key_off[KO], col_off[VO];
#pragma unroll
  for (int i = 0; i < KO; ++i)
    key_off[i] = HK == 16 ? ((tg * 16 + (lane & 7) + ((lane >> 4) << 3)) * WS + ((lane >> 3) & 1) * 8 + min(kstep(i), nks - 1) * 16) * 2
                          : ((tg * 8 + (lane & 7)) * WS + ((lane >> 3) & 1) * 8 + min(kstep(2 * i) + (lane >> 4), nks - 1) * 16) * 2;
#pragma unroll
  for (int n = 0; n < VO; ++n) col_off[n] = NT == 1 ? (a_row * WS + d0) * 2 : (a_row * WS + min(d0 + n * 16, p.rp - 16) + a_col) * 2;
  const uint32_t step16 = 16 * WS * 2;

  auto scores = [&](int st, int buf) {
    float acc[MS][HK / 8][4];
#pragma unroll
    for (int m = 0; m < MS; ++m)
#pragma unroll
      for (int n = 0; n < HK / 8; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;
    const uint32_t base = ukv0 + st * stage_bytes;
    if constexpr (HK == 16) {
#pragma unroll
      for (int i = 0; i < KPG; ++i) {
        uint32_t bb[4];
        ldsm4(base + key_off[i], bb);
#pragma unroll
        for (int m = 0; m < MS; ++m) {
          mma16816(acc[m][0], qf[m][i], bb[0], bb[1]);
          mma16816(acc[m][HK / 8 - 1], qf[m][i], bb[2], bb[3]);
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < KPG; i += 2) {       // eight keys, two k-steps
        uint32_t bb[4];
        ldsm4(base + key_off[i / 2], bb);
#pragma unroll
        for (int m = 0; m < MS; ++m) {
          mma16816(acc[m][0], qf[m][i], bb[0], bb[1]);
          mma16816(acc[m][0], qf[m][i + 1], bb[2], bb[3]);
        }
      }
    }
    float* dst = spart + (buf * kLtKG + kg) * M * SS + tg * HK + 2 * t4;
#pragma unroll
    for (int m = 0; m < MS; ++m)
#pragma unroll
      for (int n = 0; n < HK / 8; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h)
          *reinterpret_cast<float2*>(dst + ((m0 + m) * 16 + g + 8 * h) * SS + n * 8) = make_float2(acc[m][n][2 * h], acc[m][n][2 * h + 1]);
  };
  auto softmax = [&](int t, int buf) {
    float s[KPT], mx = mrun;
#pragma unroll
    for (int u = 0; u < KPT; ++u) s[u] = 0.f;
#pragma unroll
    for (int k = 0; k < kLtKG; ++k) {
      float f[KPT];
      const float* row = spart + ((buf * kLtKG + k) * M + srow) * SS + sc;
      if constexpr (KPT == 2) {
        const float2 v = *reinterpret_cast<const float2*>(row);
        f[0] = v.x;
        f[KPT - 1] = v.y;
      } else {
        load_vec<KPT>(row, f);
      }
#pragma unroll
      for (int u = 0; u < KPT; ++u) s[u] += f[u];
    }
#pragma unroll
    for (int u = 0; u < KPT; ++u) {
      const int key = kv0 + t * TOK + sc + u;
      s[u] = key <= pos && key >= lo ? s[u] * sl2 : -INFINITY;
      mx = fmaxf(mx, s[u]);
    }
#pragma unroll
    for (int off = TPR / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    // the reference point follows the maximum only when it has grown by a factor of 2^8: the output is rarely rescaled
    mx = mx > mrun + 8.f ? mx : mrun;
    const float ref = mx == -INFINITY ? 0.f : mx, alpha = fast_exp2(mrun - ref);            // nothing seen yet: 0
    const float keep = mrun == mx ? 1.f : alpha;
    mrun = mx;
    lrun *= keep;
    __nv_bfloat16* dst = sp + (buf * M + srow) * PS + sc;
#pragma unroll
    for (int u = 0; u < KPT; ++u) {
      s[u] = fast_exp2(s[u] - ref);
      lrun += s[u];
    }
    if constexpr (KPT == 2) *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(s[0], s[KPT - 1]);
    else store_vec<KPT>(dst, s);
    if (sc == 0) salpha[buf * M + srow] = keep;
  };
  auto output = [&](int st, int buf) {
    if (d0 >= p.rp) return;
    const uint32_t ukv = ukv0 + st * stage_bytes, up = up0 + buf * M * PS * 2;
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float f0 = salpha[buf * M + m * 16 + g], f1 = salpha[buf * M + m * 16 + g + 8];
      if (__any_sync(0xffffffffu, f0 != 1.f || f1 != 1.f)) {
#pragma unroll
        for (int n = 0; n < NT; ++n) { o[m][n][0] *= f0; o[m][n][1] *= f0; o[m][n][2] *= f1; o[m][n][3] *= f1; }
      }
    }
#pragma unroll
    for (int kk = 0; kk < TOK / 16; ++kk) {
      uint32_t a[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldsm4(up + ((m * 16 + a_row) * PS + kk * 16 + a_col) * 2, a[m]);
      if constexpr (NT == 1) {
        uint32_t b0, b1;                       // one n8 tile: matrices keys 0..7 and 8..15
        asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];\n"
                     : "=r"(b0), "=r"(b1) : "r"(ukv + kk * step16 + col_off[0]) : "memory");
#pragma unroll
        for (int m = 0; m < MT; ++m) mma16816(o[m][0], a[m], b0, b1);
      } else {
#pragma unroll
        for (int n = 0; n < NT / 2; ++n) {
          uint32_t x[4];                       // columns past the latent are computed and dropped
          ldsm4t(ukv + kk * step16 + col_off[n], x);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma16816(o[m][2 * n], a[m], x[0], x[1]);
            mma16816(o[m][2 * n + 1], a[m], x[2], x[3]);
          }
        }
      }
    }
  };

  if (n_tiles > 0) {
    cp_async_wait<0>();
    __syncthreads();                           // the first S - 2 >= 2 tiles
    scores(0, 0);
    __syncthreads();
    int s_prev = 0, s_cur = 0, s_next = 1, s_in = S - 2;         // ring positions of tiles p - 1, p, p + 1 and of the one requested
    for (int t = 0; t < n_tiles; ++t) {
      const int ahead = t + S - 2;
      if (ahead < n_tiles) fetch(s_in, ahead, next);
      cp_async_commit();
      next = page_of(ahead + 1);
      scores(s_next, (t + 1) & 1);             // past the last tile: stale keys, never read
      softmax(t, t & 1);
      if (t > 0) output(s_prev, (t - 1) & 1);
      // tile t + 2 has to be here; the S - 4 requested after it need not
      if (S == 4) cp_async_wait<0>();
      else if (S == 5) cp_async_wait<1>();
      else cp_async_wait<2>();
      __syncthreads();
      s_prev = s_cur;
      s_cur = s_next;
      s_next = s_next + 1 == S ? 0 : s_next + 1;
      s_in = s_in + 1 == S ? 0 : s_in + 1;
    }
    output(s_prev, (n_tiles - 1) & 1);
  }
  cp_async_wait<0>();
  // ---- row sums, output
#pragma unroll
  for (int off = TPR / 2; off > 0; off >>= 1) lrun += __shfl_xor_sync(0xffffffffu, lrun, off);
  if (sc == 0) {
    ssum[srow] = lrun;
    if (p.splits > 1 && pos >= 0) {
      float* ml = p.part_ml + ((flat0 + srow) * p.splits + split) * 2;
      ml[0] = mrun;
      ml[1] = lrun;
    }
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = m * 16 + g + 8 * h;
      if (r0 + r >= n_flat) continue;
      const long long flat = flat0 + r;
      if (p.splits == 1) {
        const float inv = 1.f / ssum[r];       // a row sees at least itself
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

template <int KPG, int NT, int MT, int WARPS, int TOK>
static int launch_latent(LatentAttnParams<__nv_bfloat16>& p, dim3 grid, cudaStream_t st) {
  constexpr int M = 16 * MT;
  const int WS = p.rp + p.ep + 8, fixed = 2 * kLtKG * M * (TOK + 4) * 4 + 2 * M * (TOK + 8) * 2 + 3 * M * 4, stage = TOK * WS * 2;
  p.stages = (227 * 1024 - fixed) / stage;
  if (p.stages > kLtMaxStages) p.stages = kLtMaxStages;
  if (p.stages < 4) return -3;
  const int smem = fixed + p.stages * stage;
  auto k = latent_attn_kernel<KPG, NT, MT, WARPS, TOK>;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(k), smem) != cudaSuccess) return -20;
  return launch_chain(k, grid, dim3(32 * WARPS), (size_t)smem, st, p) == cudaSuccess ? 0 : -21;
}
// classes of latent and row widths: NT * 8 * WARPS columns, 16 * KPG * kLtKG numbers of a row
static int launch_latent_1(LatentAttnParams<__nv_bfloat16>& p, dim3 grid, cudaStream_t st) {
  const int W = p.rp + p.ep;
  if (p.rp <= 128 && W <= 192) return launch_latent<4, 1, 1, 16, 32>(p, grid, st);
  if (p.rp <= 256 && W <= 320) return launch_latent<6, 2, 1, 16, 32>(p, grid, st);
  if (p.rp <= 512 && W <= 576) return launch_latent<10, 4, 1, 16, 32>(p, grid, st);
  if (W <= 1088) return launch_latent<18, 16, 1, 8, 16>(p, grid, st);
  return -5;
}
static int launch_latent_2(LatentAttnParams<__nv_bfloat16>& p, dim3 grid, cudaStream_t st) {
  const int W = p.rp + p.ep;
  if (p.rp <= 128 && W <= 192) return launch_latent<3, 1, 2, 16, 32>(p, grid, st);
  if (p.rp <= 256 && W <= 320) return launch_latent<5, 2, 2, 16, 32>(p, grid, st);
  if (p.rp <= 512 && W <= 576) return launch_latent<9, 4, 2, 16, 32>(p, grid, st);
  return -5;
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
  if (rp % 16 || ep % 16 || rp > 1024 || rp + ep > 1088 || (mt != 1 && mt != 2) || block_size < 1) return -1;
  if (mt == 2 && (rp > 512 || rp + ep > 576)) return -5;         // wider rows exist with 16-row tiles
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15) return -2;
  if (splits > 1 && (!part_o || !part_ml)) return -4;
  LatentAttnParams<bf16> p = {reinterpret_cast<const bf16*>(q), reinterpret_cast<const bf16*>(cache), reinterpret_cast<bf16*>(out), part_o, part_ml,
                              block_tables, bt_ld, seq_lens, query_start_loc, row_start, tiles > 0 ? tile_seq : nullptr, tile_r0, H, rp, ep,
                              block_size, -1, window, splits < 1 ? 1 : splits, 1, scale};
  for (int k = 0; k < 20; ++k)
    if (block_size == 1 << k) p.bs_shift = k;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(tiles > 0 ? tiles : B, p.splits, tiles > 0 ? 1 : (H + 16 * mt - 1) / (16 * mt));
  const int rc = mt == 1 ? launch_latent_1(p, grid, st) : launch_latent_2(p, grid, st);
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
                               block_size, -1, window, 1, 1, scale};
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
