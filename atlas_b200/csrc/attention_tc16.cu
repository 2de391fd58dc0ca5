// Prefill (chunk) attention over the paged bf16 KV cache on the 5th-generation tensor cores: head_dim 64 or 128, 16-token
// pages, any number of query heads per kv head up to 128, causal with optional chunked visibility, sliding window, softmax
// sinks, bounded scores and a bias per head by the key's distance.
//
// One CTA per (128-row query tile, kv head); the G query heads that share the kv head are packed into the tile's rows
// (row = token * G + head; rows past G * floor(128 / G) stay unused).  The cached bytes are MMA operands as they are, so
// nothing is converted: the loader warps copy 16-byte pieces of the pages straight into the swizzled operand tiles.
//
//   warp 0       TMA load of the Q tile (3-D box: 64 dims x G heads x 128/G tokens, 128-byte swizzle)
//   warp 1       tcgen05.mma issuer (kind::f16 on bf16): S_j = Q K_j^T into one of two TMEM buffers, O += P_j V_j
//   warps 2, 3   K loaders: cp.async into a ring of two 128-token tiles (rows = tokens)
//   warps 4, 5   V loaders: the same for V^T (rows = head dims); pieces past the sequence's end are zeroed
//   warps 6..13  softmax, two threads per query row (see attention_tc.cu): scores are scaled into the exp2 domain in fp32, P
//                goes to shared memory in bf16 as the A operand of the PV product, O is rescaled in TMEM lazily
//
// Key tiles before a query tile's first visible key are never loaded.  Every wait is bounded (status word + early exit).
#include "common.cuh"
#include "host_api.h"
#include "tc_util.cuh"

namespace atlas {

constexpr int kT16Rows = 128, kT16Kv = 128, kT16Page = 16, kT16Pages = kT16Kv / kT16Page, kT16Threads = 448;
constexpr int kT16Sub = 16 * 1024;            // 128 rows x 64 bf16

struct Tc16Params {
  __nv_bfloat16* out; long long ldo;
  const __nv_bfloat16* k_cache; const __nv_bfloat16* v_cache;
  const int* block_tables; int bt_ld;
  const int* seq_lens; const int* query_start_loc;
  const int* tile_seq; const int* tile_q0;
  const float* sinks;
  float scale_log2;
  float cap_in, cap_out;                      // bounded scores (cap_out 0 = off)
  const float* distance; int reach;           // [Hq, reach + 1] joins a score by the key's distance (null = off)
  int bias_ld;                                // > 0: the group's rows fit in shared memory, this many floats apart (exp2 domain)
  int Hkv, G, chunk, window;
  status_t* status;
};

// first position a row at `pos` can see
ATLAS_DEVICE int first_visible16(const Tc16Params& p, int pos) {
  const int lo = p.chunk > 0 ? pos - pos % p.chunk : 0;
  return p.window > 0 ? max(lo, pos - p.window + 1) : lo;
}

ATLAS_DEVICE void cp16(uint32_t dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
}
ATLAS_DEVICE void cp_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N>
ATLAS_DEVICE void cp_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

template <int D>
__global__ void __launch_bounds__(kT16Threads, 1)
attn_prefill_tc16_kernel(const __grid_constant__ CUtensorMap tmap_q, const Tc16Params p) {
  constexpr int NS = D / 64;                  // 64-dim sub-tiles of Q and K
  constexpr int kVSub = D * 128;              // V^T sub-tile: D rows x 64 tokens
  constexpr int kKTile = NS * kT16Sub, kVTile = 2 * kVSub;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sP = sQ + NS * kT16Sub;            // 2 sub-tiles: [128 rows][64 tokens]
  uint8_t* sK = sP + 2 * kT16Sub;             // two slots
  uint8_t* sV = sK + 2 * kKTile;              // two slots
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + 2 * kVTile);
  uint64_t* q_full = bars;
  uint64_t* k_ready = bars + 1;               // [2] 2 loader warps
  uint64_t* k_free = bars + 3;                // [2] commit after QK
  uint64_t* v_ready = bars + 5;               // [2] 2 loader warps
  uint64_t* v_free = bars + 7;                // [2] commit after PV
  uint64_t* pv_done = bars + 9;               // commit after PV: P tile free, O stable
  uint64_t* s_full = bars + 10;               // [2] commit after QK
  uint64_t* s_free = bars + 12;               // [2] 8 softmax warps
  uint64_t* p_ready = bars + 14;              // 8 softmax warps
  uint64_t* x_ready = bars + 15;              // [2 parities][4 row groups]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 23);
  volatile uint32_t* abort_flag = tmem_slot + 1;
  float* s_bias = reinterpret_cast<float*>(bars + 32);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = p.G, tpt = kT16Rows / G;      // query tokens per tile
  const int b = p.tile_seq[blockIdx.x], q0 = p.tile_q0[blockIdx.x], kvh = blockIdx.y;
  const int L = p.seq_lens[b];
  const int q_row0 = p.query_start_loc[b];
  const int q_len = p.query_start_loc[b + 1] - q_row0;
  const int ctx0 = L - q_len;
  const int first_pos = ctx0 + q0;
  const int kv_hi = min(L, ctx0 + min(q0 + tpt, q_len));         // causal bound of the tile's last live token
  const int kv_lo = first_visible16(p, first_pos) / kT16Kv * kT16Kv;
  const int n_kv = (kv_hi - kv_lo + kT16Kv - 1) / kT16Kv;        // at least 1: the tile's first token sees itself

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&k_ready[s], 2); mbar_init(&k_free[s], 1); mbar_init(&v_ready[s], 2); mbar_init(&v_free[s], 1);
      mbar_init(&s_full[s], 1); mbar_init(&s_free[s], 8);
    }
    mbar_init(pv_done, 1); mbar_init(p_ready, 8);
    for (int s = 0; s < 8; ++s) mbar_init(&x_ready[s], 2);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 512); tmem_relinquish(); }
  if (warp == 0 && lane == 0) tma_prefetch_desc(&tmap_q);
  if (p.bias_ld > 0) {
    const float* src = p.distance + (long long)kvh * G * (p.reach + 1);
    for (int g = 0; g < G; ++g)
      for (int i = threadIdx.x; i <= p.reach; i += kT16Threads) s_bias[g * p.bias_ld + i] = src[g * (p.reach + 1) + i] * 1.4426950408889634f;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tS = tmem_base, tO = tmem_base + 256, tX = tmem_base + 384;
  const int* bt = p.block_tables + (long long)b * p.bt_ld;

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(q_full, (uint32_t)(NS * 128 * G * tpt));
#pragma unroll
      for (int s = 0; s < NS; ++s) tma_load_3d(sQ + s * kT16Sub, &tmap_q, q_full, s * 64, kvh * G, q_row0 + q0);
      mbar_wait(q_full, 0, abort_flag, p.status, 0x8a0);         // the copy has landed before this warp leaves
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t kIdS = make_idesc(kT16Rows, kT16Kv, 1u), kIdO = make_idesc(kT16Rows, D, 1u);
      const uint32_t aQ = smem_u32(sQ), aK = smem_u32(sK), aV = smem_u32(sV), aP = smem_u32(sP);
      bool ok = mbar_wait(q_full, 0, abort_flag, p.status, 0x8b0);
      auto issue_pv = [&](int i) -> bool {
        const int s = i & 1;
        if (!mbar_wait(p_ready, i & 1, abort_flag, p.status, 0x8b1)) return false;
        if (!mbar_wait(&v_ready[s], (i >> 1) & 1, abort_flag, p.status, 0x8b2)) return false;
        tc_fence_after();
#pragma unroll
        for (int ks = 0; ks < kT16Kv / 16; ++ks) {
          const uint64_t ad = make_smem_desc_sw128(aP + (ks >> 2) * kT16Sub) + 2 * (ks & 3);
          const uint64_t bd = make_smem_desc_sw128(aV + s * kVTile + (ks >> 2) * kVSub) + 2 * (ks & 3);
          umma_f16(tO, ad, bd, kIdO, (i > 0 || ks > 0) ? 1u : 0u);
        }
        umma_commit(pv_done);
        umma_commit(&v_free[s]);
        return true;
      };
      for (int j = 0; j < n_kv && ok; ++j) {
        const int s = j & 1;
        if (!mbar_wait(&k_ready[s], (j >> 1) & 1, abort_flag, p.status, 0x8b3)) { ok = false; break; }
        if (!mbar_wait(&s_free[s], ((j >> 1) & 1) ^ 1u, abort_flag, p.status, 0x8b4)) { ok = false; break; }
        tc_fence_after();
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {
          const uint64_t ad = make_smem_desc_sw128(aQ + (ks >> 2) * kT16Sub) + 2 * (ks & 3);
          const uint64_t bd = make_smem_desc_sw128(aK + s * kKTile + (ks >> 2) * kT16Sub) + 2 * (ks & 3);
          umma_f16(tS + s * 128, ad, bd, kIdS, ks > 0 ? 1u : 0u);
        }
        umma_commit(&s_full[s]);
        umma_commit(&k_free[s]);
        if (j > 0) ok = issue_pv(j - 1);
      }
      if (ok) issue_pv(n_kv - 1);
    }
  } else if (warp < 6) {
    // ------------------------------------------------------------------ loaders: 64 threads for K, 64 for V
    const bool is_k = warp < 4;
    const int t = threadIdx.x - (is_k ? 64 : 128);
    uint64_t* ready = is_k ? k_ready : v_ready;
    uint64_t* freed = is_k ? k_free : v_free;
    const int n_pages = (L + kT16Page - 1) / kT16Page;
    constexpr int CPR = D / 8;                // 16-byte pieces of a K row
    for (int j = 0; j < n_kv; ++j) {
      const int s = j & 1, kv0 = kv_lo + j * kT16Kv, pg0 = kv0 / kT16Page;
      const int blk = (lane < kT16Pages && pg0 + lane < n_pages) ? bt[pg0 + lane] : 0;
      const bool go = j < 2 || mbar_wait(&freed[s], ((j - 2) >> 1) & 1, abort_flag, p.status, is_k ? 0x8c0 : 0x8c1);
      if (!__all_sync(0xffffffffu, go)) break;               // the whole warp leaves together
      if (is_k) {
        const uint32_t dst = smem_u32(sK + s * kKTile);
#pragma unroll 8
        for (int it = 0; it < kT16Kv * CPR / 64; ++it) {
          const int i = it * 64 + t, trow = i / CPR, c = i % CPR, pg = trow / kT16Page;
          const long long base = ((long long)__shfl_sync(0xffffffffu, blk, pg) * p.Hkv + kvh) * (kT16Page * D);
          cp16(dst + (c >> 3) * kT16Sub + (trow >> 3) * 1024 + (trow & 7) * 128 + (((c & 7) ^ (trow & 7)) << 4),
               p.k_cache + base + (trow % kT16Page) * D + c * 8, pg0 + pg < n_pages);
        }
      } else {
        uint8_t* tile = sV + s * kVTile;
#pragma unroll 8
        for (int it = 0; it < kT16Pages * 2 * D / 64; ++it) {
          const int i = it * 64 + t, pg = i / (2 * D), r = (i % (2 * D)) >> 1, h2 = i & 1;
          const int t0 = kv0 + pg * kT16Page + h2 * 8;
          const long long base = ((long long)__shfl_sync(0xffffffffu, blk, pg) * p.Hkv + kvh) * (kT16Page * D);
          const __nv_bfloat16* src = p.v_cache + base + r * kT16Page + h2 * 8;
          uint8_t* dst = tile + (pg >> 2) * kVSub + (r >> 3) * 1024 + (r & 7) * 128 + ((((pg & 3) * 2 + h2) ^ (r & 7)) << 4);
          if (t0 < L && t0 + 8 > L) {         // the sequence ends inside this piece: what follows may be stale
            uint4 v = *reinterpret_cast<const uint4*>(src);
            uint16_t* e = reinterpret_cast<uint16_t*>(&v);
#pragma unroll
            for (int q = 0; q < 8; ++q)
              if (t0 + q >= L) e[q] = 0;
            *reinterpret_cast<uint4*>(dst) = v;
          } else {
            cp16(smem_u32(dst), src, t0 < L);
          }
        }
      }
      cp_commit();
      if (j > 0) {
        cp_wait<1>();                         // tile j - 1 has landed
        fence_proxy_async();
        __syncwarp();
        if (lane == 0) mbar_arrive(&ready[(j - 1) & 1]);
      }
    }
    cp_wait<0>();
    fence_proxy_async();
    __syncwarp();
    if (lane == 0) mbar_arrive(&ready[(n_kv - 1) & 1]);
  } else {
    // ------------------------------------------------------------------ softmax, two threads per query row
    const int lane_group = warp & 3, half = (warp - 6) >> 2;      // score columns [64 half, + 64), output columns [D/2 half, + D/2)
    const int col0 = half * 64, ocol0 = half * (D / 2);
    constexpr int OC = D / 64;                                    // 32-column pieces of this thread's output half
    const int row = lane_group * 32 + lane;
    const uint32_t t_lane = (uint32_t)(lane_group * 32) << 16;
    bool ok = true;
    int xn = 0;
    // one value to the other thread of the same row through a TMEM column (the pair's barrier orders it)
    auto exchange = [&](float mine, float& other) -> bool {
      const int par = xn & 1;
      uint64_t* xb = &x_ready[par * 4 + lane_group];
      tmem_st_32x32b_x1(tX + t_lane + par * 2 + half, __float_as_uint(mine));
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(xb);
      const bool got = mbar_wait(xb, (xn >> 1) & 1, abort_flag, p.status, 0x8d3);
      if (!__all_sync(0xffffffffu, got)) return false;
      tc_fence_after();
      uint32_t o;
      tmem_ld_32x32b_x1(tX + t_lane + par * 2 + (half ^ 1), o);
      tmem_ld_wait();
      other = __uint_as_float(o);
      ++xn;
      return true;
    };
    auto wait_all = [&](uint64_t* bar, uint32_t parity, uint32_t site) -> bool {
      const bool got = mbar_wait(bar, parity, abort_flag, p.status, site);
      return __all_sync(0xffffffffu, got);
    };
    const int tok = q0 + row / G;
    const bool row_live = row < G * tpt && tok < q_len;
    const int pos = ctx0 + tok;
    const int lo_pos = first_visible16(p, pos);
    const bool capped = p.cap_out > 0.f;
    const bool biased = p.distance != nullptr;
    const float s_mul = capped || biased ? 1.f : p.scale_log2;
    const int bias_head = row % G;
    const float* bias_row = biased ? (p.bias_ld > 0 ? s_bias + bias_head * p.bias_ld : p.distance + (long long)(kvh * G + bias_head) * (p.reach + 1)) : nullptr;
    const float bias_mul = p.bias_ld > 0 ? 1.f : 1.4426950408889634f;
    const float bias_far = biased ? bias_row[p.reach] * bias_mul : 0.f;
    float m = -INFINITY, l = 0.f;                                 // m: reference point in the exp2 domain
    const int sw = row & 7;
    uint8_t* prow = sP + half * kT16Sub + (row >> 3) * 1024 + sw * 128;
    for (int j = 0; j < n_kv && ok; ++j) {
      const int sb = j & 1, kv0 = kv_lo + j * kT16Kv;
      if (!wait_all(&s_full[sb], (j >> 1) & 1, 0x8d0)) { ok = false; break; }
      tc_fence_after();
      const uint32_t ts = tS + sb * 128 + t_lane;
      const int vis = row_live ? pos + 1 - kv0 : 0, hid = lo_pos - kv0;       // visible columns [hid, vis)
      uint32_t sr[2][32];
#pragma unroll
      for (int c = 0; c < 2; ++c) tmem_ld_32x32b_x32(ts + col0 + c * 32, sr[c]);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_free[sb]);
      if (capped) {
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i) sr[c][i] = __float_as_uint(capped_score(__uint_as_float(sr[c][i]), p.cap_in, p.cap_out));
      }
      if (biased) {
        const float mul = capped ? 1.f : p.scale_log2;
        const int back = pos - kv0 - col0;                            // distance of this thread's first column
        if (__all_sync(0xffffffffu, back - 63 >= p.reach)) {
#pragma unroll
          for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int i = 0; i < 32; ++i) sr[c][i] = __float_as_uint(fmaf(__uint_as_float(sr[c][i]), mul, bias_far));
        } else {
#pragma unroll
          for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const float bv = bias_row[min(max(back - c * 32 - i, 0), p.reach)] * bias_mul;
              sr[c][i] = __float_as_uint(fmaf(__uint_as_float(sr[c][i]), mul, bv));
            }
        }
      }
      const bool full = __all_sync(0xffffffffu, vis >= col0 + 64 && hid <= col0);
      if (!full) {
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int col = col0 + c * 32 + i;
            if (col >= vis || col < hid) sr[c][i] = 0xff800000u;
          }
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int i = 0; i < 32; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sr[c][i]));
      const float mine = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      float theirs;
      if (!exchange(mine, theirs)) { ok = false; break; }
      const float mx = fmaxf(mine, theirs) * s_mul;              // a positive scale: checked by the host
      float m_new = m, alpha = 1.f;
      if (mx > m + 8.f) {
        m_new = mx;
        alpha = (m == -INFINITY) ? 0.f : fast_exp2(m - mx);
      }
      if (j > 0) {
        if (!wait_all(pv_done, (j - 1) & 1, 0x8d1)) { ok = false; break; }
        tc_fence_after();
        if (__any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll
          for (int c = 0; c < OC; ++c) {
            uint32_t r[32];
            tmem_ld_32x32b_x32(tO + t_lane + ocol0 + c * 32, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * alpha);
            tmem_st_32x32b_x32(tO + t_lane + ocol0 + c * 32, r);
          }
          tmem_st_wait();
        }
      }
      float sum4[4] = {0.f, 0.f, 0.f, 0.f};
      const float mref = (m_new == -INFINITY) ? 0.f : m_new;      // rows that see nothing yet: every p is 0
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          float e[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            e[i] = fast_exp2(fmaf(__uint_as_float(sr[c][q * 8 + i]), s_mul, -mref));
            sum4[i & 3] += e[i];
          }
          uint4 o;
          o.x = pack_bf16x2(e[0], e[1]); o.y = pack_bf16x2(e[2], e[3]); o.z = pack_bf16x2(e[4], e[5]); o.w = pack_bf16x2(e[6], e[7]);
          *reinterpret_cast<uint4*>(prow + (((c * 4 + q) ^ sw) << 4)) = o;
        }
      l = l * alpha + (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
      m = m_new;
      fence_proxy_async();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    float l_other = 0.f;
    if (ok) ok = exchange(l, l_other);
    l += l_other;
    if (ok && wait_all(pv_done, (n_kv - 1) & 1, 0x8d2)) {
      tc_fence_after();
      const int head = kvh * G + row % G;
      if (p.sinks && row_live) l += fast_exp2(p.sinks[head] * 1.4426950408889634f - m);
      const float inv = l > 0.f ? 1.f / l : 0.f;
      __nv_bfloat16* orow = p.out + (long long)(q_row0 + tok) * p.ldo + head * D + ocol0;
#pragma unroll
      for (int c = 0; c < OC; ++c) {
        uint32_t r[32];
        tmem_ld_32x32b_x32(tO + t_lane + ocol0 + c * 32, r);
        tmem_ld_wait();
        if (row_live) {
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            float f[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(r[q * 8 + i]) * inv;
            *reinterpret_cast<uint4*>(orow + c * 32 + q * 8) =
                make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

template <int D>
static int launch_tc16(const CUtensorMap& tq, const Tc16Params& p, int num_tiles, cudaStream_t st) {
  constexpr int kSmem = (D / 64) * kT16Sub + 2 * kT16Sub + 2 * (D / 64) * kT16Sub + 4 * D * 128 + 256 + 1024;
  Tc16Params pp = p;
  int bytes = kSmem;
  pp.bias_ld = 0;
  if (p.distance) {
    // rows 32 / G banks apart: the heads of a token meet different banks
    const int step = p.G < 32 ? 32 / p.G : 1, ld = (p.reach + 1 + 31) / 32 * 32 + step;
    if ((long long)kSmem + 4ll * p.G * ld <= 227 * 1024) { pp.bias_ld = ld; bytes += 4 * p.G * ld; }
  }
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(attn_prefill_tc16_kernel<D>), bytes) != cudaSuccess) return -20;
  attn_prefill_tc16_kernel<D><<<dim3(num_tiles, p.Hkv), kT16Threads, bytes, st>>>(tq, pp);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

}  // namespace atlas

using namespace atlas;

// `num_tiles` query tiles of floor(128 / G) tokens each, described by (sequence index, first query token of the tile inside
// the sequence's chunk).  Returns 1 when the shape is not covered, so that the caller can use the general kernel.
extern "C" int atlas_attn_prefill_tc16(const void* q, long long ldq, void* out, long long ldo, const void* k_cache, const void* v_cache,
                                       const int* block_tables, int bt_ld, const int* seq_lens, const int* query_start_loc,
                                       const int* tile_seq, const int* tile_q0, int num_tiles, int total_tokens, float scale, int Hq,
                                       int Hkv, int D, int block_size, int chunk, int window, const float* sinks, float softcap,
                                       const float* distance, int reach, unsigned long long* status, void* stream) {
  if (num_tiles <= 0) return 0;
  if (distance && reach < 0) return -2;
  if ((D != 64 && D != 128) || block_size != kT16Page || Hq % Hkv || Hq / Hkv > kT16Rows || !(scale > 0.f)) return 1;
  if ((reinterpret_cast<uintptr_t>(q) & 15) || (ldq % 8) || (ldo % 8) || (reinterpret_cast<uintptr_t>(out) & 15)) return 1;
  EncodeTiledFn enc = tc_encode_fn();
  if (!enc) return -10;
  const int G = Hq / Hkv;
  CUtensorMap tq;
  cuuint64_t dims[3] = {(cuuint64_t)D, (cuuint64_t)Hq, (cuuint64_t)total_tokens};
  cuuint64_t strides[2] = {(cuuint64_t)D * 2, (cuuint64_t)ldq * 2};
  cuuint32_t box[3] = {64, (cuuint32_t)G, (cuuint32_t)(kT16Rows / G)};
  cuuint32_t estr[3] = {1, 1, 1};
  if (enc(&tq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(q), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
          CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return -11;
  Tc16Params p;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.ldo = ldo;
  p.k_cache = reinterpret_cast<const __nv_bfloat16*>(k_cache); p.v_cache = reinterpret_cast<const __nv_bfloat16*>(v_cache);
  p.block_tables = block_tables; p.bt_ld = bt_ld; p.seq_lens = seq_lens; p.query_start_loc = query_start_loc;
  p.tile_seq = tile_seq; p.tile_q0 = tile_q0; p.sinks = sinks; p.scale_log2 = scale * 1.4426950408889634f;
  p.Hkv = Hkv; p.G = G; p.chunk = chunk; p.window = window; p.status = status;
  p.cap_in = p.cap_out = 0.f;
  p.distance = distance; p.reach = reach; p.bias_ld = 0;
  if (softcap > 0.f) cap_constants(scale, softcap, &p.cap_in, &p.cap_out);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return D == 64 ? launch_tc16<64>(tq, p, num_tiles, st) : launch_tc16<128>(tq, p, num_tiles, st);
}
