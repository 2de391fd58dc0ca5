// RG-LRU recurrence (gated linear recurrent unit, one state per channel) with its convolution and block-diagonal gates.
//
//   r = sigmoid(ra[b] u_b + bias), i = sigmoid(ri[b] u_b + bias), a = exp(-8 r softplus(lam)),  S = a S + sqrt(1 - a^2) i u,
//   out = S * gelu_tanh(y)
//
// The rows of a step are taken in chunks of 32 across sequence borders.  Inside a chunk every row gets (P, S) with
// state = S + P * (state ahead of the chunk): P is the product of the decays so far, and a sequence's first row sets P = 0 and
// S from its own stored state, so neither borders nor portions need work lists.
//
//   rglru_tc_kernel      bf16, one CTA per (two chunks, 128 channels of a block): convolution into a swizzled operand tile, both gates on
//                        tcgen05.mma with channels on the M side (gate matrices are stored as ready tiles, one bulk copy per
//                        64-deep slice), then every thread walks its channel along the chunk's rows straight from TMEM.  Steps of
//                        one row per sequence need no chunk logic: the kernel writes outputs and states itself
//   rglru_local_kernel   the same walk from gate sums in memory: fp32, and blocks too wide for shared memory
//   rglru_carry_kernel   state ahead of every chunk, channel by channel
//   rglru_finish_kernel  outputs, new states and snapshots
#include "common.cuh"
#include "host_api.h"
#include "tc_util.cuh"
#include "vec_io.cuh"

namespace atlas {

constexpr int kRgRows = 64, kRgChunk = 32;     // rows of a tile; rows of a chunk

template <typename T>
struct RgParams {
  const T* x; long long ldx;                   // convolution input (tensor-core form)
  const T* u; long long ldu;                   // convolution output (other form)
  const float* zr; const float* zi; long long z_row, z_block;     // gate sums: element (t, block, k) at t * z_row + block * z_block + k
  const T* y; long long ldy;                   // gate branch (null: states only)
  const T* conv_w; const T* conv_b; const T* conv_state; int taps;
  const T* tiles;                              // gate matrices [blocks, Mt, Kb, 2, 128, 64], 128-byte swizzle applied
  const float* gate_bias; const float* lam;    // [2, C], [C]
  float* h;                                    // [slots, C]
  float* P; float* S;                          // [rows, C]
  float* endP; float* endS;                    // [chunks, C]; endS becomes the state ahead of the chunk
  T* out; long long ldo;
  const int* seq_of; const int* qsl; const int* slots; const unsigned char* has;
  const int* limit; const int* snap_rows; const int* snap_slots; int snaps;
  int stages;                                  // slices of the gate matrices in flight
  int rows, C, n, commit, one_row, state_vec;  // state_vec: windows and taps of eight channels can be read 16 bytes at a time
  status_t* status;
};

ATLAS_DEVICE float rg_coef(float lam) {        // -8 softplus(lam)
  return -8.f * (fmaxf(lam, 0.f) + log1pf(expf(-fabsf(lam))));
}
ATLAS_DEVICE float approx_sqrt(float x) {
  float y;
  asm("sqrt.approx.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
// The decay a as its distance m = 1 - a from one, and the drive d = sqrt(1 - a^2) i u with 1 - a^2 = m (2 - m).  Close to one, where
// states live for thousands of rows, m keeps the digits that a rounded a loses (and would lose the same way in every row): near
// zero it is the Taylor sum of 1 - e^t.
template <bool kFast>
ATLAS_DEVICE void rg_gates(float zr, float zi, float u, float coef, float& m, float& d) {
  float t, i;
  if (kFast) {
    // both sigmoids from one reciprocal; below -60 a gate is shut
    const float er = 1.f + __expf(-fmaxf(zr, -60.f)), ei = 1.f + __expf(-fmaxf(zi, -60.f)), inv = __fdividef(1.f, er * ei);
    t = coef * (ei * inv);
    i = er * inv;
  } else {
    t = coef / (1.f + expf(-zr));
    i = 1.f / (1.f + expf(-zi));
  }
  const float near = -t * (1.f + t * 0.5f * (1.f + t * (1.f / 3.f) * (1.f + t * 0.25f * (1.f + t * 0.2f * (1.f + t * (1.f / 6.f))))));
  m = t > -0.25f ? near : 1.f - (kFast ? __expf(t) : expf(t));
  const float gain = m * (2.f - m);
  d = (kFast ? approx_sqrt(gain) : sqrtf(gain)) * i * u;
}
// a x + d
ATLAS_DEVICE float decayed(float m, float x, float d) { return fmaf(-m, x, x + d); }
// z (1 + tanh k) / 2 = z sigmoid(2 k)
template <bool kFast>
ATLAS_DEVICE float gelu_tanh1(float z) {
  const float k = -1.5957691216057308f * (z + 0.044715f * z * z * z);
  return kFast ? __fdividef(z, 1.f + __expf(fminf(k, 80.f))) : z / (1.f + expf(k));
}
ATLAS_DEVICE void unpack8(const uint4& v, float (&f)[8]) {
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w[j]));
    f[2 * j] = a.x; f[2 * j + 1] = a.y;
  }
}

// ----------------------------------------------------------------------------- gates on tensor cores
constexpr int kRgThreads = 256, kRgStage = 2 * 128 * 128, kRgMaxStages = 4;
using bf16 = __nv_bfloat16;

ATLAS_DEVICE void bulk_copy(void* smem_dst, const void* gsrc, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n" ::"r"(
                   smem_u32(smem_dst)),
               "l"(reinterpret_cast<uint64_t>(gsrc)), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

// kTaps: taps known at compile time (0 = p.taps); V: channels per access; kRows: rows of the tile, fewer than kRgRows in steps of one
// row per sequence
template <int kTaps, int V, int kRows>
__global__ void __launch_bounds__(kRgThreads, kRows < kRgRows ? 1 : 2)
rglru_tc_kernel(const RgParams<bf16> p) {
  constexpr bool kStep = kRows < kRgRows;
  constexpr int kWalk = kRows / 2, kSub = kRows * 128;
  extern __shared__ uint8_t rg_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(rg_raw) + 1023) & ~uintptr_t(1023));
  const int kb_n = (p.n + 63) >> 6;
  uint8_t* sW = smem;                          // [stages][r tile | i tile]
  uint8_t* sU = sW + p.stages * kRgStage;      // [kb_n][rows][64 channels]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sU + kb_n * kSub);
  uint64_t* full = bars;                       // [stages]
  uint64_t* empty = bars + kRgMaxStages;       // [stages]
  uint64_t* done = bars + 2 * kRgMaxStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * kRgMaxStages + 1);
  volatile uint32_t* abort_flag = tmem_slot + 1;
  int* s_rel = reinterpret_cast<int*>(bars + 16);              // [rows] row inside its sequence's portion (-1: no row)
  int* s_slot = s_rel + kRows;                                 // [rows] state slot
  int* s_live = s_slot + kRows;                                // [rows] the slot holds a state

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int mt_n = (p.n + 127) >> 7, blk = blockIdx.x / mt_n, mt = blockIdx.x % mt_n, t0 = blockIdx.y * kRows;
  if (tid == 0) {
    for (int s = 0; s < p.stages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    mbar_init(done, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 2 * kRows); tmem_relinquish(); }
  const uint8_t* wsrc = reinterpret_cast<const uint8_t*>(p.tiles) + (long long)(blk * mt_n + mt) * kb_n * kRgStage;
  if (tid == 0) {                              // the weights do not depend on the previous kernel
    for (int s = 0; s < p.stages && s < kb_n; ++s) {
      mbar_expect_tx(&full[s], kRgStage);
      bulk_copy(sW + s * kRgStage, wsrc + (long long)s * kRgStage, kRgStage, &full[s]);
    }
  }
  // so do the constants of the channel that this thread walks later
  const int half = warp >> 2, m = (warp & 3) * 32 + lane, mc = mt * 128 + m, row0 = half * kWalk;
  const bool mine = mc < p.n;
  const int mu = mine ? mc : 0;                // threads without a channel read one that exists
  const int c = blk * p.n + mu;
  const float br = p.gate_bias[c], bi = p.gate_bias[p.C + c], coef = rg_coef(p.lam[c]);
  chain_wait();
  if (tid < kRows) {
    const int t = t0 + tid;
    int rel = -1, slot = 0, live = 0;
    if (t < p.rows) {
      const int b = kStep ? t : p.seq_of[t];
      rel = kStep ? 0 : t - p.qsl[b]; slot = p.slots[b]; live = p.has[b] != 0;
    }
    s_rel[tid] = rel; s_slot[tid] = slot; s_live[tid] = live;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  chain_trigger();                             // this CTA has its TMEM: the next kernel may come in

  // ---- convolution of the block's channels, 8 per thread, into the operand tile (rows = tokens, zeros past the ends)
  {
    const int groups = kb_n * 8, want = groups * kRows / kRgThreads, seg = want >= 8 ? 8 : (want >= 4 ? 4 : 2), segs = kRows / seg;
    const int taps = kTaps > 0 ? kTaps : p.taps;
    for (int item = tid; item < groups * segs; item += kRgThreads) {
      const int g = item % groups, r0 = (item / groups) * seg, ch = g * 8;         // channel inside the block
      const int c0 = blk * p.n + ch, nv = min(8, p.n - ch);                        // live channels of the eight
      constexpr int kN = kTaps > 0 ? kTaps : 1;
      float w[kN][8], bias[8], win[kN][8];
      if (kTaps == 4 && V == 8 && p.state_vec && nv == 8) {
        unpack8(*reinterpret_cast<const uint4*>(p.conv_b + c0), bias);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          float f[8];
          unpack8(reinterpret_cast<const uint4*>(p.conv_w + (long long)c0 * 4)[i], f);
#pragma unroll
          for (int j = 0; j < 4; ++j) { w[j % kN][2 * i] = f[j]; w[j % kN][2 * i + 1] = f[4 + j]; }
        }
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          bias[i] = i < nv ? to_f32(p.conv_b[c0 + i]) : 0.f;
          if (kTaps > 0)
#pragma unroll
            for (int j = 0; j < kN; ++j) w[j][i] = i < nv ? to_f32(p.conv_w[(long long)(c0 + i) * taps + j]) : 0.f;
        }
      }
      auto input = [&](int row, int back, float (&f)[8]) {                         // the input `back` rows before tile row `row`
        const int rel = s_rel[row];
        if (rel < 0 || nv <= 0) {
#pragma unroll
          for (int i = 0; i < 8; ++i) f[i] = 0.f;
        } else if (back <= rel) {
          const bf16* src = p.x + (long long)(t0 + row - back) * p.ldx + c0;
          if (V == 8 && nv == 8) {
            load_vec<8>(src, f);
          } else {
#pragma unroll
            for (int i = 0; i < 8; ++i) f[i] = i < nv ? to_f32(src[i]) : 0.f;
          }
        } else {
          const bool live = s_live[row] != 0;
          const bf16* src = p.conv_state + ((long long)s_slot[row] * p.C + c0) * (taps - 1) + (taps - 1) - (back - rel);
#pragma unroll
          for (int i = 0; i < 8; ++i) f[i] = live && i < nv ? to_f32(src[(long long)i * (taps - 1)]) : 0.f;
        }
      };
      auto put = [&](int row, const float (&acc)[8]) {
        *reinterpret_cast<uint4*>(sU + (g >> 3) * kSub + row * 128 + (((g & 7) ^ (row & 7)) << 4)) =
            make_uint4(pack_bf16x2(acc[0], acc[1]), pack_bf16x2(acc[2], acc[3]), pack_bf16x2(acc[4], acc[5]), pack_bf16x2(acc[6], acc[7]));
      };
      if constexpr (kTaps > 0 && V == 8 && !kStep) {
        if (nv == 8 && s_rel[r0 + seg - 1] >= seg + kTaps - 2) {
          // the rows and their windows lie inside one portion: all loads in flight, then the sums
          const bf16* src = p.x + (long long)(t0 + r0 - (kTaps - 1)) * p.ldx + c0;
          uint4 raw[8 + kTaps - 1];
#pragma unroll
          for (int i = 0; i < 8 + kTaps - 1; ++i)
            if (i < seg + kTaps - 1) raw[i] = *reinterpret_cast<const uint4*>(src + (long long)i * p.ldx);
#pragma unroll
          for (int i = 0; i < kTaps - 1; ++i) unpack8(raw[i], win[i]);
#pragma unroll
          for (int row = 0; row < 8; ++row) {
            if (row >= seg) break;
            float acc[8];
            unpack8(raw[row + kTaps - 1], win[(row + kTaps - 1) % kTaps]);
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[i] = bias[i];
#pragma unroll
            for (int j = 0; j < kTaps; ++j)
#pragma unroll
              for (int i = 0; i < 8; ++i) acc[i] = fmaf(win[(row + j) % kTaps][i], w[j][i], acc[i]);
            put(r0 + row, acc);
          }
          continue;
        }
      }
      if constexpr (kTaps == 4 && V == 8 && kStep) {
        if (p.state_vec && nv == 8) {
          // one row per sequence: the window is the stored one, 24 consecutive numbers for the eight channels
          for (int rb = r0; rb < r0 + seg; rb += 2) {
            uint4 st[2][3], xv[2];
#pragma unroll
            for (int q = 0; q < 2; ++q) {
              const bool in = s_rel[rb + q] >= 0, live = in && s_live[rb + q] != 0;
              const uint4* sp = reinterpret_cast<const uint4*>(p.conv_state + ((long long)s_slot[rb + q] * p.C + c0) * 3);
#pragma unroll
              for (int i = 0; i < 3; ++i) st[q][i] = live ? sp[i] : make_uint4(0u, 0u, 0u, 0u);
              xv[q] = in ? *reinterpret_cast<const uint4*>(p.x + (long long)(t0 + rb + q) * p.ldx + c0) : make_uint4(0u, 0u, 0u, 0u);
            }
#pragma unroll
            for (int q = 0; q < 2; ++q) {
              float acc[8], f[8], old[24];
              unpack8(xv[q], f);
#pragma unroll
              for (int i = 0; i < 3; ++i) unpack8(st[q][i], *reinterpret_cast<float (*)[8]>(old + 8 * i));
              const bool in = s_rel[rb + q] >= 0;
#pragma unroll
              for (int i = 0; i < 8; ++i) {
                acc[i] = fmaf(f[i], w[kTaps - 1][i], bias[i]);
#pragma unroll
                for (int j = 0; j < kTaps - 1; ++j) acc[i] = fmaf(old[i * (kTaps - 1) + j], w[j][i], acc[i]);
                acc[i] = in ? acc[i] : 0.f;
              }
              put(rb + q, acc);
            }
          }
          continue;
        }
      }
      for (int row = r0; row < r0 + seg; ++row) {
        float acc[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[i] = bias[i];
        if constexpr (kTaps > 0) {
          // a sequence's first row takes its window from the stored state; later rows slide it
          if (row == r0 || s_rel[row] == 0) {
#pragma unroll
            for (int j = 0; j < kN - 1; ++j) input(row, kN - 1 - j, win[j]);
          }
          input(row, 0, win[kN - 1]);
#pragma unroll
          for (int j = 0; j < kN; ++j)
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[i] = fmaf(win[j][i], w[j][i], acc[i]);
#pragma unroll
          for (int j = 0; j < kN - 1; ++j)
#pragma unroll
            for (int i = 0; i < 8; ++i) win[j][i] = win[j + 1][i];
        } else {
          for (int j = 0; j < taps; ++j) {
            float f[8];
            input(row, taps - 1 - j, f);
#pragma unroll
            for (int i = 0; i < 8; ++i) acc[i] = fmaf(f[i], i < nv ? to_f32(p.conv_w[(long long)(c0 + i) * taps + j]) : 0.f, acc[i]);
          }
        }
        if (s_rel[row] < 0) {
#pragma unroll
          for (int i = 0; i < 8; ++i) acc[i] = 0.f;
        }
        put(row, acc);
      }
    }
  }
  fence_proxy_async();
  __syncthreads();

  // ---- gate sums: D[channel, row] of both gates, K = the block's channels
  const uint32_t tmem = *tmem_slot;
  if (tid == 0) {
    constexpr uint32_t kId = make_idesc(128, kRows, 1u);
    bool ok = true;
    for (int k = 0; k < kb_n && ok; ++k) {
      const int s = k % p.stages;
      ok = mbar_wait(&full[s], (k / p.stages) & 1, abort_flag, p.status, 0xa10);
      if (!ok) break;
      tc_fence_after();
      const uint32_t aw = smem_u32(sW + s * kRgStage), bu = smem_u32(sU + k * kSub);
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        const uint64_t bd = make_smem_desc_sw128(bu) + 2 * ks;
        umma_f16(tmem, make_smem_desc_sw128(aw) + 2 * ks, bd, kId, (k > 0 || ks > 0) ? 1u : 0u);
        umma_f16(tmem + kRows, make_smem_desc_sw128(aw + 128 * 128) + 2 * ks, bd, kId, (k > 0 || ks > 0) ? 1u : 0u);
      }
      if (k + p.stages < kb_n) {
        umma_commit(&empty[s]);
        ok = mbar_wait(&empty[s], (k / p.stages) & 1, abort_flag, p.status, 0xa11);
        if (!ok) break;
        mbar_expect_tx(&full[s], kRgStage);
        bulk_copy(sW + s * kRgStage, wsrc + (long long)(k + p.stages) * kRgStage, kRgStage, &full[s]);
      }
    }
    umma_commit(done);
  }
  __syncwarp();
  // ---- every thread walks one channel along half of the rows, eight at a time
  constexpr int kG = 8;
  const uint8_t* ucol = sU + (mu >> 6) * kSub + (mu & 7) * 2;
  const int upiece = (mu & 63) >> 3;
  auto input = [&](int row) { return to_f32(*reinterpret_cast<const bf16*>(ucol + row * 128 + ((upiece ^ (row & 7)) << 4))); };
  float hv[kG];
  bf16 yv[kG];
  auto fetch = [&](int g) {                    // one row per sequence: states and gate branch of a group of rows
#pragma unroll
    for (int j = 0; j < kG; ++j) {
      const int row = row0 + g * kG + j;
      const bool in = mine && s_rel[row] >= 0;
      hv[j] = in && s_live[row] ? p.h[(long long)s_slot[row] * p.C + c] : 0.f;
      yv[j] = in ? p.y[(long long)(t0 + row) * p.ldy + c] : __float2bfloat16_rn(0.f);
    }
  };
  if (kStep) fetch(0);
  const bool got = mbar_wait(done, 0, abort_flag, p.status, 0xa12);
  const bool all = __syncthreads_and(got ? 1 : 0) != 0;
  tc_fence_after();

  if (all) {
    const uint32_t ta = tmem + ((uint32_t)((warp & 3) * 32) << 16) + row0;
    const bool smooth = !kStep && s_rel[row0 + kWalk - 1] >= kWalk;      // all rows follow a row of the same portion
    float P = 1.f, S = 0.f;
#pragma unroll 1
    for (int g = 0; g < kWalk / kG; ++g) {
      if (s_rel[row0 + g * kG] < 0) break;     // no rows from here on
      uint32_t r[kG], q[kG];
      tmem_ld_32x32b_x8(ta + g * kG, r);
      tmem_ld_32x32b_x8(ta + kRows + g * kG, q);
      tmem_ld_wait();
      float dm[kG], d[kG];
#pragma unroll
      for (int j = 0; j < kG; ++j)
        rg_gates<true>(__uint_as_float(r[j]) + br, __uint_as_float(q[j]) + bi, input(row0 + g * kG + j), coef, dm[j], d[j]);
      const long long t = t0 + row0 + g * kG;
      if constexpr (kStep) {
#pragma unroll
        for (int j = 0; j < kG; ++j) {
          const int row = row0 + g * kG + j;
          if (!mine || s_rel[row] < 0) continue;
          const float s = decayed(dm[j], hv[j], d[j]);
          if (p.commit) p.h[(long long)s_slot[row] * p.C + c] = s;
          p.out[(t + j) * p.ldo + c] = from_f32<bf16>(s * gelu_tanh1<true>(to_f32(yv[j])));
        }
        if (g + 1 < kWalk / kG) fetch(g + 1);
      } else if (smooth) {
#pragma unroll
        for (int j = 0; j < kG; ++j) {
          S = decayed(dm[j], S, d[j]);
          P = decayed(dm[j], P, 0.f);
          if (mine) {
            p.P[(t + j) * p.C + c] = P;
            p.S[(t + j) * p.C + c] = S;
          }
        }
      } else {
#pragma unroll
        for (int j = 0; j < kG; ++j) {
          const int row = row0 + g * kG + j, rel = s_rel[row];
          if (rel < 0 || !mine) continue;
          if (rel == 0) {
            S = s_live[row] ? decayed(dm[j], p.h[(long long)s_slot[row] * p.C + c], d[j]) : d[j];
            P = 0.f;
          } else {
            S = decayed(dm[j], S, d[j]);
            P = decayed(dm[j], P, 0.f);
          }
          p.P[(t + j) * p.C + c] = P;
          p.S[(t + j) * p.C + c] = S;
        }
      }
    }
    if (!kStep && mine && s_rel[row0] >= 0) {
      const long long chunk = blockIdx.y * (kRows / kWalk) + half;
      p.endP[chunk * p.C + c] = P;
      p.endS[chunk * p.C + c] = S;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 2 * kRows);
  }
}

// ----------------------------------------------------------------------------- gate sums from memory
template <typename T>
__global__ void __launch_bounds__(128)
rglru_local_kernel(const RgParams<T> p) {
  chain_trigger();
  chain_wait();
  const int c = blockIdx.x * 128 + threadIdx.x, chunk = blockIdx.y;
  if (c >= p.C) return;
  const long long zo = (long long)(c / p.n) * p.z_block + c % p.n;
  const float br = p.gate_bias[c], bi = p.gate_bias[p.C + c], coef = rg_coef(p.lam[c]);
  float P = 1.f, S = 0.f;
  const int t1 = min(p.rows, (chunk + 1) * kRgChunk);
  for (int t = chunk * kRgChunk; t < t1; ++t) {
    const int b = p.seq_of[t];
    float dm, d;
    rg_gates<false>(p.zr[zo + t * p.z_row] + br, p.zi[zo + t * p.z_row] + bi, to_f32(p.u[t * p.ldu + c]), coef, dm, d);
    if (t == p.qsl[b]) {
      S = p.has[b] ? decayed(dm, p.h[(long long)p.slots[b] * p.C + c], d) : d;
      P = 0.f;
    } else {
      S = decayed(dm, S, d);
      P = decayed(dm, P, 0.f);
    }
    p.P[(long long)t * p.C + c] = P;
    p.S[(long long)t * p.C + c] = S;
  }
  p.endP[(long long)chunk * p.C + c] = P;
  p.endS[(long long)chunk * p.C + c] = S;
}

// ----------------------------------------------------------------------------- carries and outputs
// 32 channels per CTA, sixteen runs of up to sixteen chunks side by side
constexpr int kCarryRuns = 16, kCarryLen = 16;
__global__ void __launch_bounds__(32 * kCarryRuns)
rglru_carry_kernel(const float* __restrict__ endP, float* endS, int chunks, int C) {
  __shared__ float sp[kCarryRuns][32], ss[kCarryRuns][32], ahead[32];
  chain_trigger();
  chain_wait();
  const int lane = threadIdx.x & 31, run = threadIdx.x >> 5, c = blockIdx.x * 32 + lane;
  const bool live = c < C;
  if (run == 0) ahead[lane] = 0.f;
  for (int k0 = 0; k0 < chunks; k0 += kCarryRuns * kCarryLen) {
    const int first = k0 + run * kCarryLen;
    float P[kCarryLen], S[kCarryLen];
#pragma unroll
    for (int i = 0; i < kCarryLen; ++i) {
      const bool in = live && first + i < chunks;
      P[i] = in ? endP[(long long)(first + i) * C + c] : 1.f;
      S[i] = in ? endS[(long long)(first + i) * C + c] : 0.f;
    }
    float rp = 1.f, rs = 0.f;                  // the run as one step
#pragma unroll
    for (int i = 0; i < kCarryLen; ++i) { rs = fmaf(P[i], rs, S[i]); rp *= P[i]; }
    sp[run][lane] = rp;
    ss[run][lane] = rs;
    __syncthreads();
    float carry = ahead[lane];
    for (int j = 0; j < run; ++j) carry = fmaf(sp[j][lane], carry, ss[j][lane]);
    const float out = fmaf(rp, carry, rs);
#pragma unroll
    for (int i = 0; i < kCarryLen; ++i) {
      if (live && first + i < chunks) endS[(long long)(first + i) * C + c] = carry;
      carry = fmaf(P[i], carry, S[i]);
    }
    __syncthreads();
    if (run == kCarryRuns - 1) ahead[lane] = out;
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
rglru_finish_kernel(const RgParams<T> p) {
  chain_trigger();
  chain_wait();
  const long long t = blockIdx.x;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= p.C) return;
  float P[V], S[V], in[V];
  load_vec<V>(p.P + t * p.C + c, P);
  load_vec<V>(p.S + t * p.C + c, S);
  load_vec<V>(p.endS + (t / kRgChunk) * p.C + c, in);
#pragma unroll
  for (int i = 0; i < V; ++i) S[i] = fmaf(P[i], in[i], S[i]);
  if (p.y) {
    float y[V];
    load_vec<V>(p.y + t * p.ldy + c, y);
#pragma unroll
    for (int i = 0; i < V; ++i) y[i] = S[i] * gelu_tanh1<sizeof(T) == 2>(y[i]);
    store_vec<V>(p.out + t * p.ldo + c, y);
  }
  const int b = p.seq_of[t], rel = (int)t - p.qsl[b], len = p.qsl[b + 1] - p.qsl[b];
  if (p.commit && rel == (p.limit ? p.limit[b] : len) - 1) store_vec<V>(p.h + (long long)p.slots[b] * p.C + c, S);
  for (int s = 0; s < p.snaps; ++s) {
    const int at = p.snap_rows[b * p.snaps + s];
    if (at > 0 && rel == at - 1) store_vec<V>(p.h + (long long)p.snap_slots[b * p.snaps + s] * p.C + c, S);
  }
}

template <int kTaps, int kRows>
static int launch_tc(RgParams<bf16> p, bool vec, cudaStream_t st) {
  const int kb = (p.n + 63) / 64, mt = (p.n + 127) / 128;
  const int fixed = 1024 + kb * kRows * 128 + 128 + 3 * kRows * 4;
  // steps of one row per sequence fetch all slices they can at once; longer ones leave room for a second CTA
  p.stages = kRows < kRgRows ? kRgMaxStages : 2;
  while (p.stages > 2 && fixed + p.stages * kRgStage > 227 * 1024) --p.stages;
  const int bytes = fixed + p.stages * kRgStage;
  if (bytes > 227 * 1024) return 1;
  auto k = vec ? rglru_tc_kernel<kTaps, 8, kRows> : rglru_tc_kernel<kTaps, 1, kRows>;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(k), bytes) != cudaSuccess) return -20;
  const dim3 grid((p.C / p.n) * mt, (p.rows + kRows - 1) / kRows);
  return launch_chain_if(p.rows <= 256, k, grid, dim3(kRgThreads), (size_t)bytes, st, p) == cudaSuccess ? 0 : -21;
}

template <typename T>
static int finish(const RgParams<T>& p, cudaStream_t st) {
  const int chunks = (p.rows + kRgChunk - 1) / kRgChunk;
  launch_chain_if(p.rows <= 256, rglru_carry_kernel, dim3((p.C + 31) / 32), dim3(32 * kCarryRuns), 0, st, (const float*)p.endP, p.endS, chunks, p.C);
  const bool vec = p.C % 4 == 0 && vec_ok<T, 4>(p.y, p.ldy) && vec_ok<T, 4>(p.out, p.ldo);
  if (vec) launch_chain_if(p.rows <= 256, rglru_finish_kernel<T, 4>, dim3(p.rows, (p.C + 1023) / 1024), dim3(256), 0, st, p);
  else launch_chain_if(p.rows <= 256, rglru_finish_kernel<T, 1>, dim3(p.rows, (p.C + 255) / 256), dim3(256), 0, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

}  // namespace atlas

using namespace atlas;

template <typename T>
static RgParams<T> rg_params(const AtlasRglru* a) {
  RgParams<T> p = {};
  p.x = reinterpret_cast<const T*>(a->x); p.ldx = a->ldx; p.u = reinterpret_cast<const T*>(a->u); p.ldu = a->ldu;
  p.zr = a->zr; p.zi = a->zi; p.z_row = a->z_row; p.z_block = a->z_block; p.y = reinterpret_cast<const T*>(a->y); p.ldy = a->ldy;
  p.conv_w = reinterpret_cast<const T*>(a->conv_w); p.conv_b = reinterpret_cast<const T*>(a->conv_b);
  p.conv_state = reinterpret_cast<const T*>(a->conv_state); p.taps = a->taps; p.tiles = reinterpret_cast<const T*>(a->tiles);
  p.gate_bias = a->gate_bias; p.lam = a->lam; p.h = a->h; p.P = a->P; p.S = a->S; p.endP = a->endP; p.endS = a->endS;
  p.out = reinterpret_cast<T*>(a->out); p.ldo = a->ldo; p.seq_of = a->seq_of; p.qsl = a->qsl; p.slots = a->slots; p.has = a->has;
  p.limit = a->limit; p.snap_rows = a->snap_rows; p.snap_slots = a->snap_slots; p.snaps = a->snaps;
  p.rows = a->rows; p.C = a->C; p.n = a->n; p.commit = a->commit; p.one_row = a->one_row; p.status = a->status;
  return p;
}

// bf16: convolution, gates and recurrence of the step's rows.  one_row: every sequence brings one row, outputs and states are
// written at once; otherwise P, S [rows, C] and endP, endS [chunks, C] are scratch.  Returns 1 (nothing launched) when a block is too wide.
extern "C" int atlas_rglru_tc(const AtlasRglru* a, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->n < 1 || a->C % a->n || a->taps < 1 || a->taps > 16 || !a->tiles || (reinterpret_cast<uintptr_t>(a->tiles) & 15)) return -1;
  if (a->one_row ? (!a->y || !a->out || a->limit || a->snaps) : (!a->P || !a->S || !a->endP || !a->endS)) return -2;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  RgParams<bf16> p = rg_params<bf16>(a);
  const bool vec = a->n % 8 == 0 && vec_ok<bf16, 8>(p.x, p.ldx);
  const uintptr_t at = reinterpret_cast<uintptr_t>(p.conv_state) | reinterpret_cast<uintptr_t>(p.conv_w) | reinterpret_cast<uintptr_t>(p.conv_b);
  p.state_vec = p.C % 8 == 0 && (at & 15) == 0 ? 1 : 0;
  if (p.one_row) {
    if (p.taps != 4) return launch_tc<0, 16>(p, vec, st);
    return p.rows <= 64 ? launch_tc<4, 16>(p, vec, st) : launch_tc<4, 32>(p, vec, st);
  }
  const int rc = p.taps == 4 ? launch_tc<4, kRgRows>(p, vec, st) : launch_tc<0, kRgRows>(p, vec, st);
  if (rc) return rc;
  return finish<bf16>(p, st);
}

// the same from the convolution's output and the gate sums (no bias yet): fp32 (f32 = 1) or bf16
extern "C" int atlas_rglru_scan(const AtlasRglru* a, int f32, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->n < 1 || a->C % a->n || !a->P || !a->S || !a->endP || !a->endS || !a->zr || !a->zi) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid((a->C + 127) / 128, (a->rows + kRgChunk - 1) / kRgChunk);
  if (f32) {
    RgParams<float> p = rg_params<float>(a);
    launch_chain_if(p.rows <= 256, rglru_local_kernel<float>, grid, dim3(128), 0, st, p);
    return finish<float>(p, st);
  }
  RgParams<bf16> p = rg_params<bf16>(a);
  launch_chain_if(p.rows <= 256, rglru_local_kernel<bf16>, grid, dim3(128), 0, st, p);
  return finish<bf16>(p, st);
}
