// 32-bit attention: rotation + paged cache write and attention over an fp32 cache, for models served in float32.
//
//   rope_kv_write_f32_kernel  one warp per (token, head of q | k | v): head norms of q and k, then rotates q in place and k on
//                             its way into the cache
//   attn_f32_kernel           one warp per (query row, head), prompt rows and decode rows alike: 32 keys a step, one per
//                             lane, online softmax, then every lane accumulates its own output dimensions.  Sliding window,
//                             chunked visibility, softmax sinks, bounded scores and distance bias as in paged_attn_kernel
//                             (attention.cu).
//
// Cache layout: K [blocks, Hkv, block_size, D], V [blocks, Hkv, D, block_size].
#include "common.cuh"
#include "host_api.h"

namespace atlas {

__global__ void __launch_bounds__(128)
rope_kv_write_f32_kernel(float* q, long long ldq, const float* __restrict__ k, long long ldk, const float* __restrict__ v, long long ldv,
                         const int* __restrict__ positions, const float* __restrict__ rope, float* k_cache, float* v_cache,
                         const int* __restrict__ slot_mapping, int T, int Hq, int Hkv, int D, int rotary, int block_size,
                         const float* __restrict__ q_norm, const float* __restrict__ k_norm, int norm_dim, int plus_one, float eps) {
  extern __shared__ float sm[];                 // [4 warps][D]
  chain_trigger();
  chain_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads = Hq + 2 * Hkv;
  const long long unit = (long long)blockIdx.x * 4 + warp;
  if (unit >= (long long)T * heads) return;
  const int t = (int)(unit / heads), h = (int)(unit % heads);
  const bool is_q = h < Hq, is_k = !is_q && h < Hq + Hkv;
  const int hh = is_q ? h : (is_k ? h - Hq : h - Hq - Hkv);
  const float* src = is_q ? q + t * ldq + hh * D : (is_k ? k + t * ldk + hh * D : v + t * ldv + hh * D);
  const int slot = slot_mapping[t];
  if (!is_q && slot < 0) return;
  float* buf = sm + warp * D;
  for (int d = lane; d < D; d += 32) buf[d] = src[d];
  const float* nw = is_q ? q_norm : (is_k ? k_norm : nullptr);
  if (nw) {
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) ss += buf[d] * buf[d];
    const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)norm_dim + eps);
    for (int d = lane; d < D; d += 32) buf[d] = buf[d] * rstd * (plus_one ? 1.f + nw[d] : nw[d]);
  }
  __syncwarp();
  const int half = rotary >> 1;
  const float* cs = rope + (long long)positions[t] * rotary;
  const long long blk = is_q ? 0 : slot / block_size;
  const int off = is_q ? 0 : slot % block_size;
  for (int d = lane; d < D; d += 32) {
    float o = buf[d];
    if ((is_q || is_k) && d < rotary)
      o = d < half ? buf[d] * cs[d] - buf[d + half] * cs[half + d] : buf[d] * cs[d - half] + buf[d - half] * cs[d];
    if (is_q) q[t * ldq + hh * D + d] = o;
    else if (is_k) k_cache[((blk * Hkv + hh) * block_size + off) * D + d] = o;
    else v_cache[((blk * Hkv + hh) * D + d) * block_size + off] = o;
  }
}

struct AttnF32Params {
  const float* q; long long ldq;
  float* out; long long ldo;
  const float* k_cache; const float* v_cache;
  const int* block_tables; int bt_ld;
  const int* seq_lens; const int* query_start_loc;
  const float* sinks;
  const float* distance; int reach;            // [Hq, reach + 1] by the key's distance (null = off)
  int B, T, Hq, Hkv, block_size, window, chunk;
  float scale, softcap;
};

template <int D>
__global__ void __launch_bounds__(128)
attn_f32_kernel(const AttnF32Params p) {
  __shared__ float sq[4][D];
  constexpr int ND = D / 32;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long unit = (long long)blockIdx.x * 4 + warp;
  if (unit >= (long long)p.T * p.Hq) return;
  const int t = (int)(unit / p.Hq), head = (int)(unit % p.Hq), kvh = head / (p.Hq / p.Hkv);
  int lo_b = 0, hi_b = p.B;                     // the sequence that owns row t
  while (lo_b + 1 < hi_b) {
    const int mid = (lo_b + hi_b) >> 1;
    if (p.query_start_loc[mid] <= t) lo_b = mid; else hi_b = mid;
  }
  const int b = lo_b;
  const int pos = p.seq_lens[b] - (p.query_start_loc[b + 1] - t);
  if (pos < 0) return;                          // padding row
  int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  if (p.chunk > 0) lo = max(lo, pos - pos % p.chunk);
  for (int d = lane; d < D; d += 32) sq[warp][d] = p.q[t * p.ldq + head * D + d] * p.scale;
  __syncwarp();
  const int* bt = p.block_tables + (long long)b * p.bt_ld;
  const int bs = p.block_size;
  float m = p.sinks ? p.sinks[head] : -INFINITY, l = p.sinks ? 1.f : 0.f;
  float o[ND];
#pragma unroll
  for (int i = 0; i < ND; ++i) o[i] = 0.f;
  for (int j0 = lo - lo % 32; j0 <= pos; j0 += 32) {
    const int j = j0 + lane;
    const bool ok = j >= lo && j <= pos;
    float s = -INFINITY;
    if (ok) {
      const float4* kr = reinterpret_cast<const float4*>(p.k_cache + (((long long)bt[j / bs] * p.Hkv + kvh) * bs + j % bs) * D);
      s = 0.f;
#pragma unroll 4
      for (int d = 0; d < D / 4; ++d) {
        const float4 kv = __ldg(kr + d);
        s += kv.x * sq[warp][d * 4] + kv.y * sq[warp][d * 4 + 1] + kv.z * sq[warp][d * 4 + 2] + kv.w * sq[warp][d * 4 + 3];
      }
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      if (p.distance) s += __ldg(p.distance + (long long)head * (p.reach + 1) + min(pos - j, p.reach));
    }
    const float top = fmaxf(m, warp_max(s));
    const float f = m == -INFINITY ? 0.f : expf(m - top);
    const float e = ok ? expf(s - top) : 0.f;
    l = l * f + warp_sum(e);
    m = top;
#pragma unroll
    for (int i = 0; i < ND; ++i) o[i] *= f;
    const int jl = max(lo, j0), jh = min(pos, j0 + 31);
    for (int jj = jl; jj <= jh; ++jj) {
      const float w = __shfl_sync(0xffffffffu, e, jj - j0);
      const float* vp = p.v_cache + ((long long)bt[jj / bs] * p.Hkv + kvh) * (long long)D * bs + jj % bs;
#pragma unroll
      for (int i = 0; i < ND; ++i) o[i] = fmaf(w, __ldg(vp + (long long)(i * 32 + lane) * bs), o[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < ND; ++i) p.out[t * p.ldo + head * D + i * 32 + lane] = o[i] / l;
}

}  // namespace atlas

using namespace atlas;

extern "C" int atlas_rope_kv_write_f32(float* q, long long ldq, const float* k, long long ldk, const float* v, long long ldv,
                                       const int* positions, const float* rope, float* k_cache, float* v_cache,
                                       const int* slot_mapping, int T, int Hq, int Hkv, int D, int rotary, int block_size,
                                       const float* q_norm, const float* k_norm, int norm_dim, int plus_one, float eps, void* stream) {
  if (T <= 0) return 0;
  if (rotary > D || rotary % 2 || D > 1024) return -1;
  const long long units = (long long)T * (Hq + 2 * Hkv);
  launch_chain_if(T <= 256, rope_kv_write_f32_kernel, dim3((unsigned)((units + 3) / 4)), dim3(128), 4 * D * sizeof(float),
                  reinterpret_cast<cudaStream_t>(stream), q, ldq, k, ldk, v, ldv, positions, rope, k_cache, v_cache, slot_mapping, T, Hq,
                  Hkv, D, rotary, block_size, q_norm, k_norm, norm_dim, plus_one, eps);
  return cudaGetLastError() == cudaSuccess ? 0 : -20;
}

// rows of all B sequences of the step: prompt portions and decode rows alike
extern "C" int atlas_attn_f32(const float* q, long long ldq, float* out, long long ldo, const float* k_cache, const float* v_cache,
                              const int* block_tables, int bt_ld, const int* seq_lens, const int* query_start_loc, int B, int T,
                              float scale, int Hq, int Hkv, int D, int block_size, int window, int chunk, const float* sinks,
                              float softcap, const float* distance, int reach, void* stream) {
  if (T <= 0 || B <= 0) return 0;
  if (Hq % Hkv || block_size < 1 || (distance && reach < 0)) return -1;
  AttnF32Params p = {q, ldq, out, ldo, k_cache, v_cache, block_tables, bt_ld, seq_lens, query_start_loc, sinks, distance, reach, B, T, Hq, Hkv,
                     block_size, window, chunk, scale, softcap};
  const dim3 grid((unsigned)(((long long)T * Hq + 3) / 4));
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (D == 64) attn_f32_kernel<64><<<grid, 128, 0, st>>>(p);
  else if (D == 128) attn_f32_kernel<128><<<grid, 128, 0, st>>>(p);
  else if (D == 256) attn_f32_kernel<256><<<grid, 128, 0, st>>>(p);
  else return -2;
  return cudaGetLastError() == cudaSuccess ? 0 : -20;
}
