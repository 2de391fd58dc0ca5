// Query / key norm over all heads of a token, rotation, query temperature and the paged cache write in one pass.
//
//   row_norm_kv_kernel   one CTA per token: sums of squares of the whole query row and of the whole key row (or those handed in,
//                        where other ranks hold some of the heads), q = q / rms * w, k = k / rms * w in fp32, the first `rotary`
//                        channels of every head turned (half-split pairs), q times 1 + c ln(floor((pos + 1) / every) + 1); q is
//                        written in place, k and v to the cache.
//
// Cache layout: K [blocks, Hkv, block_size, D], V [blocks, Hkv, D, block_size], in the activations' type (bf16 or fp32).
#include "common.cuh"
#include "host_api.h"
#include "vec_io.cuh"

namespace atlas {

template <typename T>
struct RowNormParams {
  T* q; long long ldq;
  const T* k; long long ldk;
  const T* v; long long ldv;
  const int* positions; const float* rope;     // rotation table [*, rotary]: cos half, sin half
  const int* seq_positions;
  const float* qw; const float* kw;            // [Hq * D], [Hkv * D]
  const float* sums;                           // [T, 2] or null
  T* k_cache; T* v_cache;
  const int* slot_mapping;
  int Hq, Hkv, D, rotary, block_size, nq, nk, every;
  float eps, temp;
};

template <typename T, int V>
__global__ void __launch_bounds__(256)
row_norm_kv_kernel(const RowNormParams<T> p) {
  extern __shared__ float row[];               // [(Hq + Hkv) * D]
  __shared__ float red[2][8];
  chain_trigger();
  chain_wait();
  const long long t = blockIdx.x;
  const int Q = p.Hq * p.D, K = p.Hkv * p.D, tid = threadIdx.x;
  const int slot = p.slot_mapping[t];
  const long long blk = slot >= 0 ? slot / p.block_size : 0;
  const int off = slot >= 0 ? slot % p.block_size : 0;
  float ssq = 0.f, ssk = 0.f;
  for (int e = tid * V; e < Q + K; e += 256 * V) {
    float f[V];
    load_vec<V>(e < Q ? p.q + t * p.ldq + e : p.k + t * p.ldk + (e - Q), f);
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) s += f[i] * f[i];
    store_vec<V>(row + e, f);
    if (e < Q) ssq += s; else ssk += s;
  }
  if (slot >= 0) {
    for (int e = tid * V; e < K; e += 256 * V) {
      float f[V];
      load_vec<V>(p.v + t * p.ldv + e, f);
      T* dst = p.v_cache + ((blk * p.Hkv + e / p.D) * (long long)p.D + e % p.D) * p.block_size + off;
#pragma unroll
      for (int i = 0; i < V; ++i) dst[(long long)i * p.block_size] = from_f32<T>(f[i]);
    }
  }
  ssq = warp_sum(ssq);
  ssk = warp_sum(ssk);
  if ((tid & 31) == 0) { red[0][tid >> 5] = ssq; red[1][tid >> 5] = ssk; }
  __syncthreads();
  ssq = ssk = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) { ssq += red[0][i]; ssk += red[1][i]; }
  if (p.sums) { ssq = p.sums[2 * t]; ssk = p.sums[2 * t + 1]; }
  const float heat = p.temp != 0.f ? 1.f + p.temp * logf((float)((p.seq_positions[t] + 1) / p.every + 1)) : 1.f;
  const float rq = heat / sqrtf(ssq / (float)p.nq + p.eps), rk = 1.f / sqrtf(ssk / (float)p.nk + p.eps);
  const int half = p.rotary >> 1;
  const float* cs = p.rope + (p.rotary ? (long long)p.positions[t] * p.rotary : 0);
  for (int e = tid * V; e < Q + K; e += 256 * V) {
    const bool is_q = e < Q;
    if (!is_q && slot < 0) continue;
    const float r = is_q ? rq : rk;
    const float* w = is_q ? p.qw : p.kw - Q;
    const int d0 = (is_q ? e : e - Q) % p.D, h0 = e - d0;       // first channel inside its head; the head's start
    float o[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const int d = d0 + i;
      const float a = row[e + i] * w[e + i];
      if (d < p.rotary) {
        const int pd = d < half ? d + half : d - half;
        const float b = row[h0 + pd] * w[h0 + pd];
        o[i] = r * (d < half ? a * cs[d] - b * cs[half + d] : a * cs[pd] + b * cs[d]);
      } else {
        o[i] = r * a;
      }
    }
    if (is_q) store_vec<V>(p.q + t * p.ldq + e, o);
    else store_vec<V>(p.k_cache + ((blk * p.Hkv + (e - Q) / p.D) * p.block_size + off) * p.D + d0, o);
  }
}

template <typename T>
static int launch_row_norm(const RowNormParams<T>& p, int T_, cudaStream_t st) {
  const int bytes = (p.Hq + p.Hkv) * p.D * (int)sizeof(float);
  if (bytes > 200 * 1024) return -3;
  constexpr int kV = 16 / sizeof(T);
  const bool vec = p.D % kV == 0 && vec_ok<T, kV>(p.q, p.ldq) && vec_ok<T, kV>(p.k, p.ldk) && vec_ok<T, kV>(p.v, p.ldv);
  auto k = vec ? row_norm_kv_kernel<T, kV> : row_norm_kv_kernel<T, 1>;
  if (bytes > 48 * 1024 && ensure_dynamic_smem(reinterpret_cast<const void*>(k), bytes) != cudaSuccess) return -20;
  launch_chain_if(T_ <= 256, k, dim3((unsigned)T_), dim3(256), (size_t)bytes, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

}  // namespace atlas

using namespace atlas;

template <typename T>
static int row_norm(void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const int* positions, const float* rope,
                    const int* seq_positions, const float* qw, const float* kw, const float* sums, void* k_cache, void* v_cache,
                    const int* slot_mapping, int T_, int Hq, int Hkv, int D, int rotary, int block_size, int nq, int nk, float eps, float temp,
                    int every, cudaStream_t st) {
  RowNormParams<T> p = {reinterpret_cast<T*>(q), ldq, reinterpret_cast<const T*>(k), ldk, reinterpret_cast<const T*>(v), ldv, positions, rope,
                        seq_positions, qw, kw, sums, reinterpret_cast<T*>(k_cache), reinterpret_cast<T*>(v_cache), slot_mapping, Hq, Hkv, D, rotary,
                        block_size, nq, nk, every, eps, temp};
  return launch_row_norm<T>(p, T_, st);
}

extern "C" int atlas_row_norm_kv_write(void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const int* positions,
                                       const float* rope, const int* seq_positions, const float* qw, const float* kw, const float* sums,
                                       void* k_cache, void* v_cache, const int* slot_mapping, int T, int Hq, int Hkv, int D, int rotary,
                                       int block_size, int nq, int nk, float eps, float temp, int every, int f32, void* stream) {
  if (T <= 0) return 0;
  if (rotary < 0 || rotary > D || rotary % 2 || block_size < 1 || every < 1 || nq < 1 || nk < 1) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? row_norm<float>(q, ldq, k, ldk, v, ldv, positions, rope, seq_positions, qw, kw, sums, k_cache, v_cache, slot_mapping, T, Hq, Hkv, D,
                               rotary, block_size, nq, nk, eps, temp, every, st)
             : row_norm<__nv_bfloat16>(q, ldq, k, ldk, v, ldv, positions, rope, seq_positions, qw, kw, sums, k_cache, v_cache, slot_mapping, T, Hq,
                                       Hkv, D, rotary, block_size, nq, nk, eps, temp, every, st);
}
