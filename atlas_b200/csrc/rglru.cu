// RG-LRU recurrence (gated linear recurrent unit, one state per channel) with its convolution and block-diagonal gates.
//
//   r = sigmoid(ra[b] u_b + bias), i = sigmoid(ri[b] u_b + bias), a = exp(-8 r softplus(lam)),  S = a S + sqrt(1 - a^2) i u,
//   out = S * gelu_tanh(y)
//
// The rows of a step are taken in chunks of 64 across sequence borders.  Inside a chunk every row gets (P, S) with
// state = S + P * (state ahead of the chunk): P is the product of the decays so far, and a sequence's first row sets P = 0 and
// S from its own stored state, so neither borders nor portions need work lists.
//
//   rglru_tc_kernel      bf16, one CTA per (chunk, 128 channels of a block): convolution into a swizzled operand tile, both gates on
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

constexpr int kRgRows = 64;

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
  int rows, C, n, commit, one_row;
  status_t* status;
};

ATLAS_DEVICE float rg_coef(float lam) {        // -8 softplus(lam)
  return -8.f * (fmaxf(lam, 0.f) + log1pf(expf(-fabsf(lam))));
}
// 1 - e^t for t <= 0: the Taylor sum near zero, where the difference would cancel
ATLAS_DEVICE float one_minus_exp(float t, float e) {
  const float s = -t * (1.f + t * 0.5f * (1.f + t * (1.f / 3.f) * (1.f + t * 0.25f * (1.f + t * 0.2f * (1.f + t * (1.f / 6.f))))));
  return t > -0.25f ? s : 1.f - e;
}
template <bool kFast>
ATLAS_DEVICE void rg_gates(float zr, float zi, float u, float coef, float& a, float& d) {
  if (kFast) {
    const float la = coef * __fdividef(1.f, 1.f + __expf(-zr));
    a = __expf(la);
    d = sqrtf(one_minus_exp(2.f * la, a * a)) * __fdividef(u, 1.f + __expf(-zi));
  } else {
    const float la = coef / (1.f + expf(-zr));
    a = expf(la);
    d = sqrtf(one_minus_exp(2.f * la, a * a)) * u / (1.f + expf(-zi));
  }
}
ATLAS_DEVICE float gelu_tanh1(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// ----------------------------------------------------------------------------- gates on tensor cores
constexpr int kRgThreads = 256, kRgStage = 2 * 128 * 128, kRgStages = 2, kRgSub = kRgRows * 128;
using bf16 = __nv_bfloat16;

ATLAS_DEVICE void bulk_copy(void* smem_dst, const void* gsrc, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n" ::"r"(
                   smem_u32(smem_dst)),
               "l"(reinterpret_cast<uint64_t>(gsrc)), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

template <int kTaps, int V>                    // kTaps: taps known at compile time (0 = p.taps); V: channels per access
__global__ void __launch_bounds__(kRgThreads, 2)
rglru_tc_kernel(const RgParams<bf16> p) {
  extern __shared__ uint8_t rg_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(rg_raw) + 1023) & ~uintptr_t(1023));
  const int kb_n = (p.n + 63) >> 6;
  uint8_t* sW = smem;                          // [stages][r tile | i tile]
  uint8_t* sU = sW + kRgStages * kRgStage;     // [kb_n][64 rows][64 channels]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sU + kb_n * kRgSub);
  uint64_t* full = bars;                       // [stages]
  uint64_t* empty = bars + kRgStages;          // [stages]
  uint64_t* done = bars + 2 * kRgStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * kRgStages + 1);
  volatile uint32_t* abort_flag = tmem_slot + 1;
  int* s_rel = reinterpret_cast<int*>(bars + 8);               // [64] row inside its sequence's portion (-1: no row)
  int* s_slot = s_rel + kRgRows;                                // [64] state slot
  int* s_live = s_slot + kRgRows;                               // [64] the slot holds a state
  float* s_end = reinterpret_cast<float*>(s_live + kRgRows);   // [2][128] first half's (P, S)

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int mt_n = (p.n + 127) >> 7, blk = blockIdx.x / mt_n, mt = blockIdx.x % mt_n, chunk = blockIdx.y, t0 = chunk * kRgRows;
  if (tid == 0) {
    for (int s = 0; s < kRgStages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    mbar_init(done, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 128); tmem_relinquish(); }
  const uint8_t* wsrc = reinterpret_cast<const uint8_t*>(p.tiles) + (long long)(blk * mt_n + mt) * kb_n * kRgStage;
  if (tid == 0) {                              // the weights do not depend on the previous kernel
    for (int s = 0; s < kRgStages && s < kb_n; ++s) {
      mbar_expect_tx(&full[s], kRgStage);
      bulk_copy(sW + s * kRgStage, wsrc + (long long)s * kRgStage, kRgStage, &full[s]);
    }
  }
  chain_wait();
  if (tid < kRgRows) {
    const int t = t0 + tid;
    int rel = -1, slot = 0, live = 0;
    if (t < p.rows) {
      const int b = p.seq_of[t];
      rel = t - p.qsl[b]; slot = p.slots[b]; live = p.has[b] != 0;
    }
    s_rel[tid] = rel; s_slot[tid] = slot; s_live[tid] = live;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  chain_trigger();                             // this CTA has its TMEM: the next kernel may come in

  // ---- convolution of the block's channels, 8 per thread, into the operand tile (rows = tokens, zeros past the ends)
  {
    const int groups = kb_n * 8, seg = groups >= 32 ? 8 : (groups >= 16 ? 4 : 2), segs = kRgRows / seg;
    const int taps = kTaps > 0 ? kTaps : p.taps;
    for (int item = tid; item < groups * segs; item += kRgThreads) {
      const int g = item % groups, r0 = (item / groups) * seg, ch = g * 8;         // channel inside the block
      const int c0 = blk * p.n + ch, nv = min(8, p.n - ch);                        // live channels of the eight
      constexpr int kN = kTaps > 0 ? kTaps : 1;
      float w[kN][8], bias[8], win[kN][8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        bias[i] = i < nv ? to_f32(p.conv_b[c0 + i]) : 0.f;
        if (kTaps > 0)
#pragma unroll
          for (int j = 0; j < kN; ++j) w[j][i] = i < nv ? to_f32(p.conv_w[(long long)(c0 + i) * taps + j]) : 0.f;
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
        uint8_t* dst = sU + (g >> 3) * kRgSub + row * 128 + (((g & 7) ^ (row & 7)) << 4);
        *reinterpret_cast<uint4*>(dst) =
            make_uint4(pack_bf16x2(acc[0], acc[1]), pack_bf16x2(acc[2], acc[3]), pack_bf16x2(acc[4], acc[5]), pack_bf16x2(acc[6], acc[7]));
      }
    }
  }
  fence_proxy_async();
  __syncthreads();

  // ---- gate sums: D[channel, row] of both gates, K = the block's channels
  const uint32_t tmem = *tmem_slot;
  if (tid == 0) {
    constexpr uint32_t kId = make_idesc(128, kRgRows, 1u);
    bool ok = true;
    for (int k = 0; k < kb_n && ok; ++k) {
      const int s = k % kRgStages;
      ok = mbar_wait(&full[s], (k / kRgStages) & 1, abort_flag, p.status, 0xa10);
      if (!ok) break;
      tc_fence_after();
      const uint32_t aw = smem_u32(sW + s * kRgStage), bu = smem_u32(sU + k * kRgSub);
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        const uint64_t bd = make_smem_desc_sw128(bu) + 2 * ks;
        umma_f16(tmem, make_smem_desc_sw128(aw) + 2 * ks, bd, kId, (k > 0 || ks > 0) ? 1u : 0u);
        umma_f16(tmem + kRgRows, make_smem_desc_sw128(aw + 128 * 128) + 2 * ks, bd, kId, (k > 0 || ks > 0) ? 1u : 0u);
      }
      if (k + kRgStages < kb_n) {
        umma_commit(&empty[s]);
        ok = mbar_wait(&empty[s], (k / kRgStages) & 1, abort_flag, p.status, 0xa11);
        if (!ok) break;
        mbar_expect_tx(&full[s], kRgStage);
        bulk_copy(sW + s * kRgStage, wsrc + (long long)(k + kRgStages) * kRgStage, kRgStage, &full[s]);
      }
    }
    umma_commit(done);
  }
  __syncwarp();
  const bool got = mbar_wait(done, 0, abort_flag, p.status, 0xa12);
  const bool all = __syncthreads_and(got ? 1 : 0) != 0;
  tc_fence_after();

  // ---- every thread walks one channel along 32 rows
  if (all) {
    const int half = warp >> 2, m = (warp & 3) * 32 + lane, mc = mt * 128 + m, row0 = half * 32;
    const bool mine = mc < p.n;
    const int c = blk * p.n + (mine ? mc : 0);
    uint32_t r[32], q[32];
    const uint32_t ta = tmem + ((uint32_t)((warp & 3) * 32) << 16) + row0;
    tmem_ld_32x32b_x32(ta, r);
    tmem_ld_32x32b_x32(ta + kRgRows, q);
    tmem_ld_wait();
    const float br = p.gate_bias[c], bi = p.gate_bias[p.C + c], coef = rg_coef(p.lam[c]);
    const uint8_t* ucol = sU + (mc >> 6) * kRgSub + (mc & 7) * 2;
    const int upiece = (mc & 63) >> 3;
    float P = 1.f, S = 0.f;
#pragma unroll
    for (int j = 0; j < 32; ++j) {
      const int row = row0 + j, rel = s_rel[row];
      if (rel >= 0 && mine) {
        const float u = to_f32(*reinterpret_cast<const bf16*>(ucol + row * 128 + ((upiece ^ (row & 7)) << 4)));
        float a, d;
        rg_gates<true>(__uint_as_float(r[j]) + br, __uint_as_float(q[j]) + bi, u, coef, a, d);
        if (rel == 0) {
          S = s_live[row] ? fmaf(a, p.h[(long long)s_slot[row] * p.C + c], d) : d;
          P = 0.f;
        } else {
          S = fmaf(a, S, d);
          P *= a;
        }
        if (p.one_row) {
          const long long t = t0 + row;
          if (p.commit) p.h[(long long)s_slot[row] * p.C + c] = S;
          p.out[t * p.ldo + c] = from_f32<bf16>(S * gelu_tanh1(to_f32(p.y[t * p.ldy + c])));
        }
      }
      r[j] = __float_as_uint(P);
      q[j] = __float_as_uint(S);
    }
    if (!p.one_row) {
      if (half == 0) { s_end[m] = P; s_end[128 + m] = S; }
      __syncthreads();
      const float P0 = half ? s_end[m] : 1.f, S0 = half ? s_end[128 + m] : 0.f;
      if (mine) {
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          const long long t = t0 + row0 + j;
          if (t >= p.rows) break;
          const float Pj = __uint_as_float(r[j]);
          p.P[t * p.C + c] = Pj * P0;
          p.S[t * p.C + c] = fmaf(Pj, S0, __uint_as_float(q[j]));
        }
        if (half) {
          p.endP[(long long)chunk * p.C + c] = P * P0;
          p.endS[(long long)chunk * p.C + c] = fmaf(P, S0, S);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 128);
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
  const int t1 = min(p.rows, (chunk + 1) * kRgRows);
  for (int t = chunk * kRgRows; t < t1; ++t) {
    const int b = p.seq_of[t];
    float a, d;
    rg_gates<false>(p.zr[zo + t * p.z_row] + br, p.zi[zo + t * p.z_row] + bi, to_f32(p.u[t * p.ldu + c]), coef, a, d);
    if (t == p.qsl[b]) {
      S = p.has[b] ? fmaf(a, p.h[(long long)p.slots[b] * p.C + c], d) : d;
      P = 0.f;
    } else {
      S = fmaf(a, S, d);
      P *= a;
    }
    p.P[(long long)t * p.C + c] = P;
    p.S[(long long)t * p.C + c] = S;
  }
  p.endP[(long long)chunk * p.C + c] = P;
  p.endS[(long long)chunk * p.C + c] = S;
}

// ----------------------------------------------------------------------------- carries and outputs
__global__ void __launch_bounds__(64)
rglru_carry_kernel(const float* __restrict__ endP, float* endS, int chunks, int C) {
  chain_trigger();
  chain_wait();
  const int c = blockIdx.x * 64 + threadIdx.x;
  if (c >= C) return;
  constexpr int kB = 16;
  float carry = 0.f;
  for (int k0 = 0; k0 < chunks; k0 += kB) {
    float P[kB], S[kB];
#pragma unroll
    for (int i = 0; i < kB; ++i) {
      const bool in = k0 + i < chunks;
      P[i] = in ? endP[(long long)(k0 + i) * C + c] : 0.f;
      S[i] = in ? endS[(long long)(k0 + i) * C + c] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < kB; ++i) {
      if (k0 + i < chunks) endS[(long long)(k0 + i) * C + c] = carry;
      carry = fmaf(P[i], carry, S[i]);
    }
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
  load_vec<V>(p.endS + (t / kRgRows) * p.C + c, in);
#pragma unroll
  for (int i = 0; i < V; ++i) S[i] = fmaf(P[i], in[i], S[i]);
  if (p.y) {
    float y[V];
    load_vec<V>(p.y + t * p.ldy + c, y);
#pragma unroll
    for (int i = 0; i < V; ++i) y[i] = S[i] * gelu_tanh1(y[i]);
    store_vec<V>(p.out + t * p.ldo + c, y);
  }
  const int b = p.seq_of[t], rel = (int)t - p.qsl[b], len = p.qsl[b + 1] - p.qsl[b];
  if (p.commit && rel == (p.limit ? p.limit[b] : len) - 1) store_vec<V>(p.h + (long long)p.slots[b] * p.C + c, S);
  for (int s = 0; s < p.snaps; ++s) {
    const int at = p.snap_rows[b * p.snaps + s];
    if (at > 0 && rel == at - 1) store_vec<V>(p.h + (long long)p.snap_slots[b * p.snaps + s] * p.C + c, S);
  }
}

template <int kTaps>
static int launch_tc(const RgParams<bf16>& p, bool vec, cudaStream_t st) {
  const int kb = (p.n + 63) / 64, mt = (p.n + 127) / 128;
  const int bytes = 1024 + kRgStages * kRgStage + kb * kRgSub + 64 + 3 * kRgRows * 4 + 2 * 128 * 4;
  if (bytes > 227 * 1024) return 1;
  auto k = vec ? rglru_tc_kernel<kTaps, 8> : rglru_tc_kernel<kTaps, 1>;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(k), bytes) != cudaSuccess) return -20;
  const dim3 grid((p.C / p.n) * mt, (p.rows + kRgRows - 1) / kRgRows);
  return launch_chain_if(p.rows <= 256, k, grid, dim3(kRgThreads), (size_t)bytes, st, p) == cudaSuccess ? 0 : -21;
}

template <typename T>
static int finish(const RgParams<T>& p, cudaStream_t st) {
  const int chunks = (p.rows + kRgRows - 1) / kRgRows;
  launch_chain_if(p.rows <= 256, rglru_carry_kernel, dim3((p.C + 63) / 64), dim3(64), 0, st, (const float*)p.endP, p.endS, chunks, p.C);
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
  const int rc = p.taps == 4 ? launch_tc<4>(p, vec, st) : launch_tc<0>(p, vec, st);
  if (rc || p.one_row) return rc;
  return finish<bf16>(p, st);
}

// the same from the convolution's output and the gate sums (no bias yet): fp32 (f32 = 1) or bf16
extern "C" int atlas_rglru_scan(const AtlasRglru* a, int f32, void* stream) {
  if (a->rows <= 0) return 0;
  if (a->n < 1 || a->C % a->n || !a->P || !a->S || !a->endP || !a->endS || !a->zr || !a->zi) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid((a->C + 127) / 128, (a->rows + kRgRows - 1) / kRgRows);
  if (f32) {
    RgParams<float> p = rg_params<float>(a);
    launch_chain_if(p.rows <= 256, rglru_local_kernel<float>, grid, dim3(128), 0, st, p);
    return finish<float>(p, st);
  }
  RgParams<bf16> p = rg_params<bf16>(a);
  launch_chain_if(p.rows <= 256, rglru_local_kernel<bf16>, grid, dim3(128), 0, st, p);
  return finish<bf16>(p, st);
}
