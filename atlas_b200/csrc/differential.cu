// Differential attention around the paged attention kernels (two maps per head over the same values):
//
//   map_norm_kv_kernel     RMS norm and rotation (half-split pairs) of every map of q and k in fp32.  Keys go to the cache as
//                          [map 1 | map 2], values beside them; the query of map m becomes a row of the cache width with zeros where the
//                          other map's key lies.  Blocks of the first kind take maps (a group of lanes each), those of the second kind
//                          turn the values of 16 tokens around for the transposed value pages.
//   map_difference_kernel  o = a_1 - lam a_2, RMS norm over the head's dv numbers, times `rest` and the sigmoid of a gate
//
// Cache layout: K [blocks, G, block_size, D], V [blocks, G, D, block_size], in the activations' type (bf16 or fp32).
#include "common.cuh"
#include "host_api.h"
#include "vec_io.cuh"

namespace atlas {

constexpr int kMapThreads = 256;
constexpr int kValueTokens = 16;              // tokens of a value block
constexpr int kMaxMap = 256, kValuePitch = kMaxMap + 4;

template <typename T>
struct MapNormParams {
  const T* q; long long ldq;                  // [T, H, 2, dim]
  const T* k; long long ldk;                  // [T, G, 2, dim]
  const T* v; long long ldv;                  // [T, G, dv]
  T* rows;                                    // [T, 2 H, D]
  const int* positions; const float* rope;    // rotation table [*, rotary]: cos half, sin half
  const float* qw; const float* kw;           // [dim]
  T* k_cache; T* v_cache;
  const int* slot_mapping;
  int T_, H, G, dim, dv, D, rotary, block_size;
  int map_blocks;                             // blocks of the first kind
  int lanes;                                  // vector form: lanes of a map, a power of two
  int vec_v;                                  // values can be read eight at a time
  float eps;
};

template <typename T>
ATLAS_DEVICE void write_values(const MapNormParams<T>& p, int vb, T* sm) {
  const int g = vb % p.G, t0 = vb / p.G * kValueTokens, n = min(kValueTokens, p.T_ - t0);
  if (p.vec_v) {
    const int pieces = p.dv / 8;
    for (int i = threadIdx.x; i < n * pieces; i += kMapThreads) {
      const int t = i / pieces, e = i % pieces * 8;
      float f[8];
      load_vec<8>(p.v + (t0 + t) * p.ldv + g * p.dv + e, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) sm[t * kValuePitch + e + j] = from_f32<T>(f[j]);
    }
  } else {
    for (int i = threadIdx.x; i < n * p.dv; i += kMapThreads) sm[i / p.dv * kValuePitch + i % p.dv] = p.v[(t0 + i / p.dv) * p.ldv + g * p.dv + i % p.dv];
  }
  // sixteen neighbouring places of a page that start on a vector boundary
  const int first = p.slot_mapping[t0];
  bool run = n == kValueTokens && first >= 0 && first % kValueTokens == 0;
  if (threadIdx.x < (unsigned)n) run = run && p.slot_mapping[t0 + threadIdx.x] == first + (int)threadIdx.x;
  run = __syncthreads_and(run);
  if (run) {
    T* dst = p.v_cache + ((long long)(first / p.block_size) * p.G + g) * p.D * p.block_size + first % p.block_size;
    for (int e = threadIdx.x; e < p.dv; e += kMapThreads) {
      float f[kValueTokens];
#pragma unroll
      for (int t = 0; t < kValueTokens; ++t) f[t] = to_f32(sm[t * kValuePitch + e]);
      store_vec<kValueTokens>(dst + (long long)e * p.block_size, f);
    }
    return;
  }
  for (int i = threadIdx.x; i < n * p.dv; i += kMapThreads) {
    const int t = i / p.dv, e = i % p.dv, slot = p.slot_mapping[t0 + t];
    if (slot >= 0) p.v_cache[(((long long)(slot / p.block_size) * p.G + g) * p.D + e) * p.block_size + slot % p.block_size] = sm[t * kValuePitch + e];
  }
}

template <typename T, bool kVec>
__global__ void __launch_bounds__(kMapThreads)
map_norm_kv_kernel(const MapNormParams<T> p) {
  __shared__ __align__(16) float sm[kValueTokens * kValuePitch];
  chain_trigger();
  chain_wait();
  if ((int)blockIdx.x >= p.map_blocks) {
    write_values(p, (int)blockIdx.x - p.map_blocks, reinterpret_cast<T*>(sm));
    return;
  }
  const int lanes = kVec ? p.lanes : 32, lane = threadIdx.x % lanes;
  const int per_token = 2 * (p.H + p.G);
  const long long unit = (long long)blockIdx.x * (kMapThreads / lanes) + threadIdx.x / lanes;
  const bool live = unit < (long long)p.T_ * per_token;
  const long long t = live ? unit / per_token : 0;
  const int a = live ? (int)(unit % per_token) : 0;          // q maps first, then k maps
  const bool is_q = a < 2 * p.H;
  const int map = is_q ? a : a - 2 * p.H, m = map & 1;
  const T* src = is_q ? p.q + t * p.ldq + (long long)map * p.dim : p.k + t * p.ldk + (long long)map * p.dim;
  const float* w = is_q ? p.qw : p.kw;
  const int slot = is_q ? 0 : p.slot_mapping[t];
  const bool write = live && slot >= 0;
  const int half = p.rotary >> 1;
  const float* cs = p.rope + (p.rotary ? (long long)p.positions[t] * p.rotary : 0);
  T* dst = is_q ? p.rows + (t * 2 * p.H + map) * p.D + m * p.dim
                : p.k_cache + (((long long)(max(slot, 0) / p.block_size) * p.G + (map >> 1)) * p.block_size + max(slot, 0) % p.block_size) * p.D + m * p.dim;
  if constexpr (kVec) {
    // eight numbers per lane: four pairs that turn together, or eight neighbours behind the rotated part
    const bool mine = live && lane < p.dim / 8, turns = lane < p.rotary / 8;
    const int d0 = turns ? 4 * lane : p.rotary + 8 * (lane - p.rotary / 8), d1 = turns ? half + 4 * lane : d0 + 4;
    float x[4] = {}, y[4] = {};
    if (mine) {
      load_vec<4>(src + d0, x);
      load_vec<4>(src + d1, y);
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) ss += x[i] * x[i] + y[i] * y[i];
    for (int s = lanes >> 1; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
    if (!write) return;
    const float rstd = 1.f / sqrtf(ss / (float)p.dim + p.eps);
    if (mine) {
      float wx[4], wy[4];
      load_vec<4>(w + d0, wx);
      load_vec<4>(w + d1, wy);
#pragma unroll
      for (int i = 0; i < 4; ++i) { x[i] *= rstd * wx[i]; y[i] *= rstd * wy[i]; }
      if (turns) {
        float c[4], s[4];
        load_vec<4>(cs + d0, c);
        load_vec<4>(cs + half + d0, s);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float u = x[i], v = y[i];
          x[i] = u * c[i] - v * s[i];
          y[i] = v * c[i] + u * s[i];
        }
      }
      store_vec<4>(dst + d0, x);
      store_vec<4>(dst + d1, y);
    }
    if (is_q) {
      const float none[4] = {};
      T* row = dst - m * p.dim;
      for (int z = lane; z < (p.D - p.dim) / 4; z += lanes) store_vec<4>(row + (4 * z < m * p.dim ? 4 * z : 4 * z + p.dim), none);
    }
  } else {
    float* buf = sm + threadIdx.x / 32 * kMaxMap;
    float ss = 0.f;
    for (int d = lane; live && d < p.dim; d += 32) {
      const float f = to_f32(src[d]);
      buf[d] = f * w[d];
      ss += f * f;
    }
    const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
    __syncwarp();
    if (!write) return;
    for (int d = lane; d < p.dim; d += 32) {
      float o = buf[d];
      if (d < p.rotary) o = d < half ? buf[d] * cs[d] - buf[d + half] * cs[half + d] : buf[d] * cs[d - half] + buf[d - half] * cs[d];
      dst[d] = from_f32<T>(o * rstd);
    }
    if (is_q) {
      T* row = dst - m * p.dim;
      for (int z = lane; z < p.D - p.dim; z += 32) row[z < m * p.dim ? z : z + p.dim] = from_f32<T>(0.f);
    }
  }
}

template <typename T>
struct MapDifferenceParams {
  const T* a;                                 // [T, 2 H, D]
  const T* gate; long long ldg;               // [T, H * dv] or null
  T* out;                                     // [T, H * dv]
  long long units;                            // T * H
  int H, D, dv, lanes;
  float lam, rest, eps;
};

template <typename T, bool kVec>
__global__ void __launch_bounds__(256)
map_difference_kernel(const MapDifferenceParams<T> p) {
  chain_trigger();
  chain_wait();
  const int lanes = kVec ? p.lanes : 32, lane = threadIdx.x % lanes;
  const long long unit = (long long)blockIdx.x * (256 / lanes) + threadIdx.x / lanes;
  const bool live = unit < p.units;
  const long long t = live ? unit / p.H : 0;
  const int h = live ? (int)(unit % p.H) : 0;
  const T* a1 = p.a + (live ? unit : 0) * 2 * p.D;
  const T* gate = p.gate ? p.gate + t * p.ldg + (long long)h * p.dv : nullptr;
  T* out = p.out + (live ? unit : 0) * p.dv;
  float o[8] = {};
  float ss = 0.f;
  const int e = lane * 8;
  if (kVec && live && e < p.dv) {
    float second[8];
    load_vec<8>(a1 + e, o);
    load_vec<8>(a1 + p.D + e, second);
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] -= p.lam * second[i];
  }
  if (!kVec) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int d = i * 32 + lane;
      if (live && d < p.dv) o[i] = to_f32(a1[d]) - p.lam * to_f32(a1[p.D + d]);
    }
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) ss += o[i] * o[i];
  for (int s = lanes >> 1; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  const float f = p.rest / sqrtf(ss / (float)p.dv + p.eps);
  if (kVec && live && e < p.dv) {
    float g[8];
    if (gate) load_vec<8>(gate + e, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = gate ? o[i] * f * sigmoid_for<T>(g[i]) : o[i] * f;
    store_vec<8>(out + e, o);
  }
  if (!kVec) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int d = i * 32 + lane;
      if (live && d < p.dv) out[d] = from_f32<T>(gate ? o[i] * f * sigmoid_for<T>(to_f32(gate[d])) : o[i] * f);
    }
  }
}

static int lanes_for(int pieces) {
  int n = 1;
  while (n < pieces) n *= 2;
  return n;
}

template <typename T>
static int launch_map_norm(MapNormParams<T> p, cudaStream_t st) {
  const bool vec = p.dim % 8 == 0 && p.rotary % 8 == 0 && vec_ok<T, 4>(p.q, p.ldq) && vec_ok<T, 4>(p.k, p.ldk) && vec_ok<float, 4>(p.qw, 0) &&
                   vec_ok<float, 4>(p.kw, 0) && vec_ok<float, 4>(p.rope, 0);
  p.vec_v = p.dv % 8 == 0 && vec_ok<T, 8>(p.v, p.ldv);
  p.lanes = vec ? lanes_for(p.dim / 8) : 32;
  const int per_block = kMapThreads / p.lanes;
  const long long maps = (long long)p.T_ * 2 * (p.H + p.G);
  p.map_blocks = (int)((maps + per_block - 1) / per_block);
  const unsigned grid = p.map_blocks + (p.T_ + kValueTokens - 1) / kValueTokens * p.G;
  launch_chain_if(p.T_ <= 256, vec ? map_norm_kv_kernel<T, true> : map_norm_kv_kernel<T, false>, dim3(grid), dim3(kMapThreads), 0, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <typename T>
static int map_norm(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, void* rows, const int* positions,
                    const float* rope, const float* qw, const float* kw, void* k_cache, void* v_cache, const int* slot_mapping, int T_, int H, int G,
                    int dim, int dv, int D, int rotary, int block_size, float eps, cudaStream_t st) {
  MapNormParams<T> p = {reinterpret_cast<const T*>(q), ldq, reinterpret_cast<const T*>(k), ldk, reinterpret_cast<const T*>(v), ldv,
                        reinterpret_cast<T*>(rows), positions, rope, qw, kw, reinterpret_cast<T*>(k_cache), reinterpret_cast<T*>(v_cache),
                        slot_mapping, T_, H, G, dim, dv, D, rotary, block_size, 0, 0, 0, eps};
  return launch_map_norm<T>(p, st);
}

template <typename T>
static int map_difference(const void* a, const void* gate, long long ldg, void* out, int T_, int H, int D, int dv, float lam, float rest, float eps,
                          cudaStream_t st) {
  MapDifferenceParams<T> p = {reinterpret_cast<const T*>(a), reinterpret_cast<const T*>(gate), ldg, reinterpret_cast<T*>(out), (long long)T_ * H, H,
                              D, dv, 32, lam, rest, eps};
  const bool vec = dv % 8 == 0 && vec_ok<T, 8>(a, D) && vec_ok<T, 8>(gate, ldg) && vec_ok<T, 8>(out, dv);
  if (vec) p.lanes = lanes_for(dv / 8);
  const long long per_block = 256 / p.lanes;
  launch_chain_if(T_ <= 256, vec ? map_difference_kernel<T, true> : map_difference_kernel<T, false>, dim3((unsigned)((p.units + per_block - 1) / per_block)),
                  dim3(256), 0, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

}  // namespace atlas

using namespace atlas;

extern "C" int atlas_map_norm_kv_write(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, void* rows,
                                       const int* positions, const float* rope, const float* qw, const float* kw, void* k_cache, void* v_cache,
                                       const int* slot_mapping, int T, int H, int G, int dim, int dv, int D, int rotary, int block_size, float eps,
                                       int f32, void* stream) {
  if (T <= 0) return 0;
  if (dim < 1 || 2 * dim > D || dv < 1 || dv > D || D > kMaxMap || D % 4 || rotary < 0 || rotary > dim || rotary % 2 || block_size < 1 || block_size % 16)
    return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? map_norm<float>(q, ldq, k, ldk, v, ldv, rows, positions, rope, qw, kw, k_cache, v_cache, slot_mapping, T, H, G, dim, dv, D, rotary,
                               block_size, eps, st)
             : map_norm<__nv_bfloat16>(q, ldq, k, ldk, v, ldv, rows, positions, rope, qw, kw, k_cache, v_cache, slot_mapping, T, H, G, dim, dv, D,
                                       rotary, block_size, eps, st);
}

extern "C" int atlas_map_difference(const void* a, const void* gate, long long ldg, void* out, int T, int H, int D, int dv, float lam, float rest,
                                    float eps, int f32, void* stream) {
  if (T <= 0) return 0;
  if (H < 1 || dv < 1 || dv > D || D > kMaxMap) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? map_difference<float>(a, gate, ldg, out, T, H, D, dv, lam, rest, eps, st)
             : map_difference<__nv_bfloat16>(a, gate, ldg, out, T, H, D, dv, lam, rest, eps, st);
}
