// Hyper-connected residual streams (fp32), the token-shift mixes of WKV layers and gated units.
//
//   hyper_norm_kernel       one CTA per token: rewrites the S streams with the last sublayer's connection and output
//                             x'[t] = sum_s mix[s, t] * x[s] + write[t] * y
//                           reads the next sublayer's input u = sum_s read[s] * x'[s] and writes rmsnorm(u) * w.  The write
//                           of one sublayer and the read + norm of the next one share a single pass over the streams.
//                           With a second output y2 (two mixers side by side) y is half the sum of both after an RMS norm
//                           each; at the start of the model the streams are set to the scaled embedding instead.
//   token_shift_mix_kernel  out[s] = x + (x_prev - x) * mu[s] for S mixes, x_prev = the previous token's row (from the
//                           sequence's state slot for the first row of a chunk, zeros at the start of a sequence)
//   group_norm_gate_kernel  rms norm over channel groups joined with a gate: norm(y * silu(z)) * w (Mamba-2),
//                           norm(y) * w * silu(z) (WKV) or norm(y / den) * w * sigmoid(z) (mLSTM)
//   add_normed_kernel       one CTA per token: x += rmsnorm(y) * w or x += y on an fp32 residual, y being a sublayer's output or the
//                           weighted sum of expert rows (and a shared expert's row); adds a step vector where one is given and hands
//                           the new x on in the activations' dtype, normed again where asked; the rich form also gates y, takes
//                           layer norms and sums over the results of all layers so far
//   gelu_embedding_kernel   gelu_tanh(z) times a slice of a token's embedding row
//   head_gate_kernel        x[t, h, :] *= sigmoid(g[t, h])
//   gated_unit_kernel       g = min(gate, limit), u = clamp(up, +-limit):  g * sigmoid(alpha g) * (u + shift), of [gate | up] or of
//                           alternating columns
//
// Every kernel exists for bf16 and fp32 activations (template parameter T).
#include "common.cuh"
#include "host_api.h"
#include "vec_io.cuh"

namespace atlas {

template <typename T>
struct HyperParams {
  float* x;                                    // [T, S, W]
  const T* y; long long ldy;
  const T* y2; long long ldy2;
  const float* w1; const float* w2;            // [W] norm weights of y / y2
  const float* mix; const float* write; const float* read;
  const float* norm_w;
  T* out; long long ldo;
  int S, W, init, store;
  float scale, eps;
};

constexpr int kMaxStreams = 8;

ATLAS_DEVICE float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();                             // red may still be read from an earlier reduction
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) s += red[i];
  return s;
}

// kS: number of streams known at compile time (0 = p.S, at most kMaxStreams)
template <typename T, int kS, int V>
__global__ void __launch_bounds__(512)
hyper_norm_kernel(const HyperParams<T> p) {
  constexpr int kN = kS > 0 ? kS : kMaxStreams;
  extern __shared__ float su[];                // [W] the read mix
  __shared__ float red[16];
  __shared__ float cf[kMaxStreams * (kMaxStreams + 2)];
  chain_trigger();
  const int S = kS > 0 ? kS : p.S;
  const long long t = blockIdx.x;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) cf[i] = p.init ? 0.f : p.mix[i];
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    cf[S * S + i] = p.init ? p.scale : p.write[i];
    cf[S * S + S + i] = p.read[i];
  }
  chain_wait();
  const T* y = p.y + t * p.ldy;
  const T* y2 = p.y2 ? p.y2 + t * p.ldy2 : nullptr;
  float r1 = 1.f, r2 = 0.f;
  if (y2) {
    float a = 0.f, b = 0.f;
    for (int e = threadIdx.x * V; e < p.W; e += blockDim.x * V) {
      float f[V], g[V];
      load_vec<V>(y + e, f);
      load_vec<V>(y2 + e, g);
#pragma unroll
      for (int i = 0; i < V; ++i) { a += f[i] * f[i]; b += g[i] * g[i]; }
    }
    r1 = 0.5f / sqrtf(block_sum(a, red) / (float)p.W + p.eps);
    r2 = 0.5f / sqrtf(block_sum(b, red) / (float)p.W + p.eps);
  }
  __syncthreads();
  float wr[kN], rd[kN];
#pragma unroll
  for (int s = 0; s < kN; ++s)
    if (s < S) { wr[s] = cf[S * S + s]; rd[s] = cf[S * S + S + s]; }
  float* x = p.x + t * (long long)S * p.W;
  float ss = 0.f;
  for (int e = threadIdx.x * V; e < p.W; e += blockDim.x * V) {
    float yv[V];
    load_vec<V>(y + e, yv);
    if (y2) {
      float g[V], a[V], b[V];
      load_vec<V>(y2 + e, g);
      load_vec<V>(p.w1 + e, a);
      load_vec<V>(p.w2 + e, b);
#pragma unroll
      for (int i = 0; i < V; ++i) yv[i] = yv[i] * r1 * a[i] + g[i] * r2 * b[i];
    }
    float old[kN][V];
    if (!p.init) {
#pragma unroll
      for (int s = 0; s < kN; ++s)
        if (s < S) load_vec<V>(x + (long long)s * p.W + e, old[s]);
    }
    float u[V];
#pragma unroll
    for (int i = 0; i < V; ++i) u[i] = 0.f;
#pragma unroll
    for (int q = 0; q < kN; ++q) {
      if (q >= S) break;
      float n[V];
#pragma unroll
      for (int i = 0; i < V; ++i) n[i] = wr[q] * yv[i];
      if (!p.init) {
#pragma unroll
        for (int s = 0; s < kN; ++s) {
          if (s >= S) break;
          const float m = cf[s * S + q];
#pragma unroll
          for (int i = 0; i < V; ++i) n[i] = fmaf(m, old[s][i], n[i]);
        }
      }
      if (p.store) store_vec<V>(x + (long long)q * p.W + e, n);
#pragma unroll
      for (int i = 0; i < V; ++i) u[i] = fmaf(rd[q], n[i], u[i]);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) { su[e + i] = u[i]; ss += u[i] * u[i]; }
  }
  const float rstd = 1.f / sqrtf(block_sum(ss, red) / (float)p.W + p.eps);
  for (int e = threadIdx.x * V; e < p.W; e += blockDim.x * V) {
    float w[V], o[V];
    load_vec<V>(p.norm_w + e, w);
#pragma unroll
    for (int i = 0; i < V; ++i) o[i] = su[e + i] * rstd * w[i];
    store_vec<V>(p.out + t * p.ldo + e, o);
  }
}

template <typename T, int V>
static int launch_hyper(const HyperParams<T>& p, int rows, cudaStream_t st) {
  const int smem = p.W * (int)sizeof(float);
  int threads = 128;
  while (threads < 512 && threads * V < p.W) threads *= 2;
  void (*k)(const HyperParams<T>) = nullptr;
  switch (p.S) {
    case 1: k = hyper_norm_kernel<T, 1, V>; break;
    case 2: k = hyper_norm_kernel<T, 2, V>; break;
    case 3: k = hyper_norm_kernel<T, 3, V>; break;
    case 4: k = hyper_norm_kernel<T, 4, V>; break;
    default: k = hyper_norm_kernel<T, 0, V>; break;
  }
  if (smem > 40 * 1024 && ensure_dynamic_smem(reinterpret_cast<const void*>(k), smem) != cudaSuccess) return -20;
  launch_chain_if(rows <= 256, k, dim3(rows), dim3(threads), smem, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <typename T>
static int hyper_norm(float* x, int rows, int S, int W, const void* y, long long ldy, const void* y2, long long ldy2,
                      const float* w1, const float* w2, const float* mix, const float* write, const float* read,
                      const float* norm_w, void* out, long long ldo, int init, int store, float scale, float eps, cudaStream_t st) {
  HyperParams<T> p;
  p.x = x; p.y = reinterpret_cast<const T*>(y); p.ldy = ldy; p.y2 = reinterpret_cast<const T*>(y2); p.ldy2 = ldy2;
  p.w1 = w1; p.w2 = w2; p.mix = mix; p.write = write; p.read = read; p.norm_w = norm_w;
  p.out = reinterpret_cast<T*>(out); p.ldo = ldo; p.S = S; p.W = W; p.init = init; p.store = store; p.scale = scale; p.eps = eps;
  const bool vec = W % 4 == 0 && vec_ok<T, 4>(y, ldy) && vec_ok<T, 4>(y2, ldy2) && vec_ok<T, 4>(out, ldo) &&
                   vec_ok<float, 4>(x, 0) && vec_ok<float, 4>(norm_w, 0) && vec_ok<float, 4>(w1, 0) && vec_ok<float, 4>(w2, 0);
  return vec ? launch_hyper<T, 4>(p, rows, st) : launch_hyper<T, 1>(p, rows, st);
}

// ----------------------------------------------------------------------------- token shift
constexpr int kShiftRows = 8;                  // consecutive rows of one thread (1 for few rows): mu and the previous row stay in registers

template <typename T, int S, int V, int R>
__global__ void __launch_bounds__(256)
token_shift_mix_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ mu, const T* __restrict__ shift,
                       const int* __restrict__ seq_of_token, const int* __restrict__ query_start_loc,
                       const int* __restrict__ state_slots, const unsigned char* __restrict__ has_state, T* out, int rows, int W) {
  chain_trigger();
  chain_wait();
  const int e = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (e >= W) return;
  float m[S][V];
#pragma unroll
  for (int s = 0; s < S; ++s) load_vec<V>(mu + (long long)s * W + e, m[s]);
  const int t0 = blockIdx.x * R, t1 = min(rows, t0 + R);
  float prev[V];
  for (int t = t0; t < t1; ++t) {
    const int b = seq_of_token[t];
    if (t == query_start_loc[b]) {
      if (has_state[b]) {
        load_vec<V>(shift + (long long)state_slots[b] * W + e, prev);
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) prev[i] = 0.f;
      }
    } else if (t == t0) {
      load_vec<V>(x + (long long)(t - 1) * ldx + e, prev);
    }
    float c[V];
    load_vec<V>(x + (long long)t * ldx + e, c);
#pragma unroll
    for (int s = 0; s < S; ++s) {
      float o[V];
#pragma unroll
      for (int i = 0; i < V; ++i) o[i] = fmaf(prev[i] - c[i], m[s][i], c[i]);
      store_vec<V>(out + ((long long)s * rows + t) * W + e, o);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) prev[i] = c[i];
  }
}

template <typename T, int V>
static int launch_shift(const void* x, long long ldx, const float* mu, const void* shift, const int* seq, const int* qsl,
                        const int* slots, const unsigned char* has, void* out, int rows, int W, cudaStream_t st) {
  const unsigned gy = (W + 256 * V - 1) / (256 * V);
  if (rows <= 256)
    launch_chain_if(true, token_shift_mix_kernel<T, 5, V, 1>, dim3(rows, gy), dim3(256), 0, st, reinterpret_cast<const T*>(x), ldx, mu,
                    reinterpret_cast<const T*>(shift), seq, qsl, slots, has, reinterpret_cast<T*>(out), rows, W);
  else
    launch_chain_if(false, token_shift_mix_kernel<T, 5, V, kShiftRows>, dim3((rows + kShiftRows - 1) / kShiftRows, gy), dim3(256), 0, st,
                    reinterpret_cast<const T*>(x), ldx, mu, reinterpret_cast<const T*>(shift), seq, qsl, slots, has,
                    reinterpret_cast<T*>(out), rows, W);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

// ----------------------------------------------------------------------------- gated group norm
// TPG threads per (row, group): a quarter of a warp for head-sized groups, a warp, or a whole block for wide ones
// kGate: 0 silu before the norm, 1 silu after it, 2 sigmoid after it.  `den` [rows, groups] (may be null): divisor of the group.
enum { kSiluFirst = 0, kSiluAfter = 1, kSigmoidAfter = 2 };
template <typename T, int TPG, int V, int kGate>
__global__ void __launch_bounds__(256)
group_norm_gate_kernel(const T* __restrict__ y, long long ldy, const T* __restrict__ z, long long ldz,
                       const float* __restrict__ w, T* out, long long ldo, int rows, int groups, int gsize, float eps,
                       const float* __restrict__ den) {
  constexpr bool kGateFirst = kGate == kSiluFirst;
  __shared__ float red[8];
  chain_trigger();
  chain_wait();
  const long long unit = (long long)blockIdx.x * (256 / TPG) + threadIdx.x / TPG;
  const bool live = unit < (long long)rows * groups;            // every lane stays for the warp's sums
  const int tid = threadIdx.x % TPG;
  const long long t = live ? unit / groups : 0;
  const int g0 = (int)(unit % groups) * gsize;
  const T* yr = y + t * ldy + g0;
  const T* zr = z + t * ldz + g0;
  const float inv = den && live ? 1.f / den[unit] : 1.f;
  float ss = 0.f;
  for (int e = tid * V; e < gsize; e += TPG * V) {
    float f[V], g[V];
    load_vec<V>(yr + e, f);
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] *= inv;
    if (kGateFirst) {
      load_vec<V>(zr + e, g);
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] *= g[i] / (1.f + expf(-g[i]));
    }
#pragma unroll
    for (int i = 0; i < V; ++i) ss += f[i] * f[i];
  }
#pragma unroll
  for (int off = (TPG < 32 ? TPG : 32) / 2; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
  if (TPG > 32) {
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += red[i];
  }
  if (!live) return;
  const float rstd = inv / sqrtf(ss / (float)gsize + eps);
  for (int e = tid * V; e < gsize; e += TPG * V) {
    float f[V], g[V], wv[V];
    load_vec<V>(yr + e, f);
    load_vec<V>(zr + e, g);
#pragma unroll
    for (int i = 0; i < V; ++i) wv[i] = w[g0 + e + i];
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = f[i] * rstd * wv[i] * ((kGate == kSigmoidAfter ? 1.f : g[i]) / (1.f + expf(-g[i])));
    store_vec<V>(out + t * ldo + g0 + e, f);
  }
}

template <typename T, int V, int kGate>
static int launch_gnorm(const void* y, long long ldy, const void* z, long long ldz, const float* w, void* out, long long ldo,
                        int rows, int groups, int gsize, float eps, const float* den, cudaStream_t st) {
  const long long units = (long long)rows * groups;
  const T *yp = reinterpret_cast<const T*>(y), *zp = reinterpret_cast<const T*>(z);
  if (gsize >= 1024)
    launch_chain_if(rows <= 256, group_norm_gate_kernel<T, 256, V, kGate>, dim3((unsigned)units), dim3(256), 0, st, yp, ldy, zp, ldz, w,
                    reinterpret_cast<T*>(out), ldo, rows, groups, gsize, eps, den);
  else if (gsize <= 128)
    launch_chain_if(rows <= 256, group_norm_gate_kernel<T, 8, V, kGate>, dim3((unsigned)((units + 31) / 32)), dim3(256), 0, st, yp, ldy,
                    zp, ldz, w, reinterpret_cast<T*>(out), ldo, rows, groups, gsize, eps, den);
  else
    launch_chain_if(rows <= 256, group_norm_gate_kernel<T, 32, V, kGate>, dim3((unsigned)((units + 7) / 8)), dim3(256), 0, st, yp, ldy,
                    zp, ldz, w, reinterpret_cast<T*>(out), ldo, rows, groups, gsize, eps, den);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <typename T, int V>
static int launch_gnorm_gate(const void* y, long long ldy, const void* z, long long ldz, const float* w, void* out, long long ldo, int rows,
                             int groups, int gsize, float eps, int kind, const float* den, cudaStream_t st) {
  if (kind == kSiluFirst) return launch_gnorm<T, V, kSiluFirst>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, den, st);
  if (kind == kSiluAfter) return launch_gnorm<T, V, kSiluAfter>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, den, st);
  return launch_gnorm<T, V, kSigmoidAfter>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, den, st);
}

template <typename T>
static int gnorm(const void* y, long long ldy, const void* z, long long ldz, const float* w, void* out, long long ldo, int rows,
                 int groups, int gsize, float eps, int kind, const float* den, cudaStream_t st) {
  if (sizeof(T) == 2 && gsize % 8 == 0 && (gsize < 1024 || gsize >= 2048) && vec_ok<T, 8>(y, ldy) && vec_ok<T, 8>(z, ldz) && vec_ok<T, 8>(out, ldo))
    return launch_gnorm_gate<T, 8>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, kind, den, st);
  const bool vec = gsize % 4 == 0 && vec_ok<T, 4>(y, ldy) && vec_ok<T, 4>(z, ldz) && vec_ok<T, 4>(out, ldo);
  if (vec) return launch_gnorm_gate<T, 4>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, kind, den, st);
  return launch_gnorm_gate<T, 1>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, kind, den, st);
}

// ----------------------------------------------------------------------------- normed outputs on an fp32 residual
template <typename T>
struct AddNormedParams {
  float* x; long long ldx;                     // [T, W]
  const T* y; long long ldy;
  const int* slot_of; const float* pick_w; int picks;      // picks > 0: y = sum_j pick_w[t, j] * rows slot_of[t, j] (>= 0) of `y`
  const T* extra; long long lde;               // joins y (null = off)
  const float* w; const float* out_w;          // w null: x += y; out_w null: out = x
  const float* step;                           // [W] added to the new x (null = off)
  T* out; long long ldo;
  int W, plus_one, store, first;               // first: x = y * scale (start of the model)
  float eps, scale;
  // kRich only
  const T* gate; long long ldg;                // y is multiplied by sigmoid(gate) first (null = off)
  const float* b; const float* out_b;          // biases: the norm with that weight is a layer norm (null = RMS norm)
  float* hist; long long hist_ld;              // results of the layers, [entries][T, W]: the new x becomes entry hist_index (null = off) ...
  const float* factors; int hist_index;        // ... and sum_j factors[j] * entry j goes on in its place (null = x itself)
};

// subtracts the row's mean from y and returns the sum of squares of what is left
template <int V, int NI>
ATLAS_DEVICE float take_mean_off(float (&y)[NI][V], int W, int step, float* red) {
  float s = 0.f;
#pragma unroll
  for (int k = 0; k < NI; ++k) {
    if (threadIdx.x * V + k * step >= W) continue;
#pragma unroll
    for (int i = 0; i < V; ++i) s += y[k][i];
  }
  const float mean = block_sum(s, red) / (float)W;
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < NI; ++k) {
    if (threadIdx.x * V + k * step >= W) continue;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      y[k][i] -= mean;
      ss += y[k][i] * y[k][i];
    }
  }
  return ss;
}

// NI pieces of V elements per thread, the row stays in registers
template <typename T, int V, int NI, bool kRich>
__global__ void __launch_bounds__(1024)
add_normed_kernel(const AddNormedParams<T> p) {
  __shared__ float red[32];
  chain_trigger();
  chain_wait();
  const long long t = blockIdx.x;
  const int step = blockDim.x * V;
  float y[NI][V];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < NI; ++k) {
    const int e = threadIdx.x * V + k * step;
#pragma unroll
    for (int i = 0; i < V; ++i) y[k][i] = 0.f;
    if (e >= p.W) continue;
    if (p.extra) load_vec<V>(p.extra + t * p.lde + e, y[k]);
    if (p.picks == 0) {
      if (p.extra) {
        float f[V];
        load_vec<V>(p.y + t * p.ldy + e, f);
#pragma unroll
        for (int i = 0; i < V; ++i) y[k][i] += f[i];
      } else {
        load_vec<V>(p.y + t * p.ldy + e, y[k]);
      }
    } else {
      for (int j = 0; j < p.picks; ++j) {
        const int row = p.slot_of[t * p.picks + j];
        if (row < 0) continue;
        const float wj = p.pick_w[t * p.picks + j];
        float f[V];
        load_vec<V>(p.y + row * p.ldy + e, f);
#pragma unroll
        for (int i = 0; i < V; ++i) y[k][i] = fmaf(wj, f[i], y[k][i]);
      }
    }
    if (kRich && p.gate) {
      float g[V];
      load_vec<V>(p.gate + t * p.ldg + e, g);
#pragma unroll
      for (int i = 0; i < V; ++i) y[k][i] *= sigmoid_for<T>(g[i]);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) ss += y[k][i] * y[k][i];
  }
  const float plus = p.plus_one ? 1.f : 0.f;
  if (p.w) {
    if (kRich && p.b) ss = take_mean_off<V, NI>(y, p.W, step, red);
    const float rstd = 1.f / sqrtf(block_sum(ss, red) / (float)p.W + p.eps);
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < NI; ++k) {
      const int e = threadIdx.x * V + k * step;
      if (e >= p.W) continue;
      float w[V], x[V];
      load_vec<V>(p.w + e, w);
      load_vec<V>(p.x + t * p.ldx + e, x);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        y[k][i] = fmaf(y[k][i] * rstd, w[i] + plus, x[i]);
        if (!(kRich && p.b)) ss += y[k][i] * y[k][i];
      }
      if (kRich && p.b) {
        float b[V];
        load_vec<V>(p.b + e, b);
#pragma unroll
        for (int i = 0; i < V; ++i) {
          y[k][i] += b[i];
          ss += y[k][i] * y[k][i];
        }
      }
    }
  } else if (!p.first || p.scale != 1.f) {
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < NI; ++k) {
      const int e = threadIdx.x * V + k * step;
      if (e >= p.W) continue;
      if (p.first) {
#pragma unroll
        for (int i = 0; i < V; ++i) y[k][i] *= p.scale;
      } else {
        float x[V];
        load_vec<V>(p.x + t * p.ldx + e, x);
#pragma unroll
        for (int i = 0; i < V; ++i) y[k][i] += x[i];
      }
#pragma unroll
      for (int i = 0; i < V; ++i) ss += y[k][i] * y[k][i];
    }
  }
  if (p.step) {
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < NI; ++k) {
      const int e = threadIdx.x * V + k * step;
      if (e >= p.W) continue;
      float f[V];
      load_vec<V>(p.step + e, f);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        y[k][i] += f[i];
        ss += y[k][i] * y[k][i];
      }
    }
  }
  if (kRich && p.hist) {
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < NI; ++k) {
      const int e = threadIdx.x * V + k * step;
      if (e >= p.W) continue;
      const float* past = p.hist + t * p.W + e;
      if (p.store) store_vec<V>(p.hist + p.hist_index * p.hist_ld + t * p.W + e, y[k]);
      if (p.factors) {
        const float own = __ldg(p.factors + p.hist_index);
#pragma unroll
        for (int i = 0; i < V; ++i) y[k][i] *= own;
#pragma unroll 4
        for (int j = 0; j < p.hist_index; ++j) {
          const float fj = __ldg(p.factors + j);
          float h[V];
          load_vec<V>(past + j * p.hist_ld, h);
#pragma unroll
          for (int i = 0; i < V; ++i) y[k][i] = fmaf(fj, h[i], y[k][i]);
        }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) ss += y[k][i] * y[k][i];
    }
  }
  if (p.store) {
#pragma unroll
    for (int k = 0; k < NI; ++k) {
      const int e = threadIdx.x * V + k * step;
      if (e < p.W) store_vec<V>(p.x + t * p.ldx + e, y[k]);
    }
  }
  if (kRich && p.out_b) ss = take_mean_off<V, NI>(y, p.W, step, red);
  const float orstd = p.out_w ? 1.f / sqrtf(block_sum(ss, red) / (float)p.W + p.eps) : 1.f;
#pragma unroll
  for (int k = 0; k < NI; ++k) {
    const int e = threadIdx.x * V + k * step;
    if (e >= p.W) continue;
    if (p.out_w) {
      float w[V];
      load_vec<V>(p.out_w + e, w);
#pragma unroll
      for (int i = 0; i < V; ++i) y[k][i] = y[k][i] * orstd * (w[i] + plus);
      if (kRich && p.out_b) {
        load_vec<V>(p.out_b + e, w);
#pragma unroll
        for (int i = 0; i < V; ++i) y[k][i] += w[i];
      }
    }
    store_vec<V>(p.out + t * p.ldo + e, y[k]);
  }
}

template <typename T>
static int add_normed(float* x, long long ldx, const void* y, long long ldy, const int* slot_of, const float* pick_w, int picks, const void* extra,
                      long long lde, const float* w, const float* out_w, const float* step, void* out, long long ldo, int rows, int W, int plus_one,
                      int store, int first, float eps, float scale, const AtlasNormedExtras& o, cudaStream_t st) {
  AddNormedParams<T> p = {x, ldx, reinterpret_cast<const T*>(y), ldy, slot_of, pick_w, picks, reinterpret_cast<const T*>(extra), lde, w, out_w, step,
                          reinterpret_cast<T*>(out), ldo, W, plus_one, store, first, eps, scale, reinterpret_cast<const T*>(o.gate), o.ldg, o.b,
                          o.out_b, o.hist, o.hist_ld, o.factors, o.hist_index};
  const bool rich = o.gate || o.b || o.out_b || o.hist;
  const bool vec = W % 8 == 0 && vec_ok<T, 8>(y, ldy) && vec_ok<T, 8>(out, ldo) && vec_ok<float, 4>(x, ldx) && vec_ok<float, 4>(w, 0) &&
                   vec_ok<float, 4>(out_w, 0) && vec_ok<float, 4>(step, 0) && vec_ok<T, 8>(extra, lde) && vec_ok<T, 8>(o.gate, o.ldg) &&
                   vec_ok<float, 4>(o.b, 0) && vec_ok<float, 4>(o.out_b, 0) && vec_ok<float, 4>(o.hist, o.hist_ld);
  const int v = vec ? 8 : 1, pieces = (W + v - 1) / v;
  void (*k)(const AddNormedParams<T>) = nullptr;
  int ni = 1;
  if (vec) {
    ni = pieces <= 1024 ? 1 : 4;
    k = ni == 1 ? (rich ? add_normed_kernel<T, 8, 1, true> : add_normed_kernel<T, 8, 1, false>)
                : (rich ? add_normed_kernel<T, 8, 4, true> : add_normed_kernel<T, 8, 4, false>);
  } else {
    ni = pieces <= 1024 ? 1 : 32;
    k = ni == 1 ? (rich ? add_normed_kernel<T, 1, 1, true> : add_normed_kernel<T, 1, 1, false>)
                : (rich ? add_normed_kernel<T, 1, 32, true> : add_normed_kernel<T, 1, 32, false>);
  }
  const int threads = ((pieces + ni - 1) / ni + 31) / 32 * 32;
  if (threads > 1024) return -2;
  launch_chain_if(rows <= 256, k, dim3(rows), dim3(threads), 0, st, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
head_gate_kernel(T* x, long long ldx, const float* __restrict__ g, long long ldg, int H, int D) {
  chain_trigger();
  chain_wait();
  const long long t = blockIdx.x;
  const int e = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (e >= H * D) return;
  const float s = 1.f / (1.f + expf(-g[t * ldg + e / D]));
  float f[V];
  load_vec<V>(x + t * ldx + e, f);
#pragma unroll
  for (int i = 0; i < V; ++i) f[i] *= s;
  store_vec<V>(x + t * ldx + e, f);
}

template <typename T, int V>
static int launch_head_gate(void* x, long long ldx, const float* g, long long ldg, int rows, int H, int D, cudaStream_t st) {
  launch_chain_if(rows <= 256, head_gate_kernel<T, V>, dim3(rows, (H * D + 256 * V - 1) / (256 * V)), dim3(256), 0, st, reinterpret_cast<T*>(x), ldx, g,
                  ldg, H, D);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

// ----------------------------------------------------------------------------- gated units, tanh
template <typename T, int V, bool kPaired>
__global__ void __launch_bounds__(256)
gated_unit_kernel(const T* __restrict__ gu, long long ld, int I, T* y, long long ldy, GatedUnit unit) {
  chain_trigger();
  chain_wait();
  const long long t = blockIdx.x;
  const int e = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (e >= I) return;
  float g[V], u[V], o[V];
  if constexpr (kPaired) {
    float f[2 * V];
    load_vec<2 * V>(gu + t * ld + 2 * e, f);
#pragma unroll
    for (int i = 0; i < V; ++i) { g[i] = f[2 * i]; u[i] = f[2 * i + 1]; }
  } else {
    load_vec<V>(gu + t * ld + e, g);
    load_vec<V>(gu + t * ld + I + e, u);
  }
#pragma unroll
  for (int i = 0; i < V; ++i) o[i] = gated_unit(g[i], u[i], unit);
  store_vec<V>(y + t * ldy + e, o);
}

template <typename T, int V, bool kPaired = false>
static int launch_glu(const void* gu, long long ld, int rows, int I, void* y, long long ldy, GatedUnit unit, cudaStream_t st) {
  dim3 grid(rows, (I + 256 * V - 1) / (256 * V));
  launch_chain_if(rows <= 256, gated_unit_kernel<T, V, kPaired>, grid, dim3(256), 0, st, reinterpret_cast<const T*>(gu), ld, I,
                  reinterpret_cast<T*>(y), ldy, unit);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

// one thread per piece of V columns of a row
template <typename T, int V>
__global__ void __launch_bounds__(256)
gelu_embedding_kernel(const T* __restrict__ z, long long ldz, const T* __restrict__ table, long long ldt, const long long* __restrict__ ids, int first,
                      int n, int N, T* out, long long ldo, int rows) {
  chain_trigger();
  chain_wait();
  const int pieces = N / V;
  const long long unit = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (unit >= (long long)rows * pieces) return;
  const long long t = unit / pieces;
  const int e = (int)(unit % pieces) * V;
  float o[V] = {};
  if (e < n) {
    float f[V];
    load_vec<V>(z + t * ldz + e, o);
    load_vec<V>(table + ids[t] * ldt + first + e, f);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float u = 0.7978845608028654f * (o[i] + 0.044715f * o[i] * o[i] * o[i]);
      o[i] = 0.5f * o[i] * (1.f + tanhf(u)) * f[i];
    }
  }
  store_vec<V>(out + t * ldo + e, o);
}

template <typename T, int V>
static int launch_gelu_embedding(const void* z, long long ldz, const void* table, long long ldt, const long long* ids, int first, int n, int N,
                                 void* out, long long ldo, int rows, cudaStream_t st) {
  const long long units = (long long)rows * (N / V);
  launch_chain_if(rows <= 256, gelu_embedding_kernel<T, V>, dim3((unsigned)((units + 255) / 256)), dim3(256), 0, st, reinterpret_cast<const T*>(z), ldz,
                  reinterpret_cast<const T*>(table), ldt, ids, first, n, N, reinterpret_cast<T*>(out), ldo, rows);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <typename T>
__global__ void __launch_bounds__(256)
tanh_kernel(T* x, long long n) {
  chain_trigger();
  chain_wait();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) x[i] = from_f32<T>(tanhf(to_f32(x[i])));
}

}  // namespace atlas

using namespace atlas;

// x [rows, S, W] fp32; y / y2 / out in bf16 (f32 = 0) or fp32 (f32 = 1)
extern "C" int atlas_hyper_norm(float* x, int rows, int S, int W, const void* y, long long ldy, const void* y2, long long ldy2,
                                const float* w1, const float* w2, const float* mix, const float* write, const float* read,
                                const float* norm_w, void* out, long long ldo, int init, int store, float scale, float eps,
                                int f32, void* stream) {
  if (rows <= 0) return 0;
  if (S < 1 || S > kMaxStreams || W < 1 || W > 50 * 1024) return -1;
  if (y2 && (!w1 || !w2 || init)) return -2;
  if (!init && (!mix || !write)) return -3;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? hyper_norm<float>(x, rows, S, W, y, ldy, y2, ldy2, w1, w2, mix, write, read, norm_w, out, ldo, init, store, scale, eps, st)
             : hyper_norm<__nv_bfloat16>(x, rows, S, W, y, ldy, y2, ldy2, w1, w2, mix, write, read, norm_w, out, ldo, init, store, scale,
                                         eps, st);
}

// five mixes: mu [5, W] fp32, out [5, rows, W]; shift [slots, W] holds every sequence's previous row
extern "C" int atlas_token_shift_mix(const void* x, long long ldx, const float* mu, const void* shift, const int* seq_of_token,
                                     const int* qsl, const int* slots, const unsigned char* has, void* out, int rows, int W,
                                     int f32, void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (f32) {
    const bool vec = W % 4 == 0 && vec_ok<float, 4>(x, ldx) && vec_ok<float, 4>(mu, 0) && vec_ok<float, 4>(shift, W) && vec_ok<float, 4>(out, W);
    return vec ? launch_shift<float, 4>(x, ldx, mu, shift, seq_of_token, qsl, slots, has, out, rows, W, st)
               : launch_shift<float, 1>(x, ldx, mu, shift, seq_of_token, qsl, slots, has, out, rows, W, st);
  }
  using B = __nv_bfloat16;
  const bool vec = W % 4 == 0 && vec_ok<B, 4>(x, ldx) && vec_ok<float, 4>(mu, 0) && vec_ok<B, 4>(shift, W) && vec_ok<B, 4>(out, W);
  return vec ? launch_shift<B, 4>(x, ldx, mu, shift, seq_of_token, qsl, slots, has, out, rows, W, st)
             : launch_shift<B, 1>(x, ldx, mu, shift, seq_of_token, qsl, slots, has, out, rows, W, st);
}

// gu: [gate | up], or alternating gate and up columns with `paired`
extern "C" int atlas_gated_unit(const void* gu, long long ld, int rows, int I, void* y, long long ldy, float limit, float alpha,
                                 float shift, int paired, int f32, void* stream) {
  if (rows <= 0 || I <= 0) return 0;
  const GatedUnit unit = {limit, alpha, shift};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (paired) {
    if (f32) {
      const bool vec = I % 4 == 0 && vec_ok<float, 4>(gu, ld) && vec_ok<float, 4>(y, ldy);
      return vec ? launch_glu<float, 4, true>(gu, ld, rows, I, y, ldy, unit, st)
                 : launch_glu<float, 1, true>(gu, ld, rows, I, y, ldy, unit, st);
    }
    using B = __nv_bfloat16;
    const bool vec = I % 8 == 0 && vec_ok<B, 8>(gu, ld) && vec_ok<B, 8>(y, ldy);
    return vec ? launch_glu<B, 8, true>(gu, ld, rows, I, y, ldy, unit, st) : launch_glu<B, 1, true>(gu, ld, rows, I, y, ldy, unit, st);
  }
  if (f32) {
    const bool vec = I % 4 == 0 && vec_ok<float, 4>(gu, ld) && vec_ok<float, 4>(y, ldy);
    return vec ? launch_glu<float, 4>(gu, ld, rows, I, y, ldy, unit, st) : launch_glu<float, 1>(gu, ld, rows, I, y, ldy, unit, st);
  }
  using B = __nv_bfloat16;
  const bool vec = I % 8 == 0 && vec_ok<B, 8>(gu, ld) && vec_ok<B, 8>(y, ldy);
  return vec ? launch_glu<B, 8>(gu, ld, rows, I, y, ldy, unit, st) : launch_glu<B, 1>(gu, ld, rows, I, y, ldy, unit, st);
}

extern "C" int atlas_tanh(void* x, long long n, int f32, void* stream) {
  if (n <= 0) return 0;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid((unsigned)((n + 255) / 256));
  if (f32) launch_chain_if(n <= 65536, tanh_kernel<float>, grid, dim3(256), 0, st, reinterpret_cast<float*>(x), n);
  else launch_chain_if(n <= 65536, tanh_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, reinterpret_cast<__nv_bfloat16*>(x), n);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

// gate_first: silu(z) before the norm; otherwise silu(z), or with `sigmoid` sigmoid(z), after it
extern "C" int atlas_group_norm_gate(const void* y, long long ldy, const void* z, long long ldz, const float* w, void* out, long long ldo,
                                     int rows, int groups, int gsize, float eps, int gate_first, int sigmoid, const float* den, int f32,
                                     void* stream) {
  if (rows <= 0) return 0;
  if (gate_first && sigmoid) return -1;
  const int kind = gate_first ? kSiluFirst : (sigmoid ? kSigmoidAfter : kSiluAfter);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? gnorm<float>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, kind, den, st)
             : gnorm<__nv_bfloat16>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, kind, den, st);
}

// fp32 residual x [rows, W]: x += rmsnorm(y) * w (w null: x += y; first: x = y * scale), then x += step (null: nothing), out = x or
// rmsnorm(x) * out_w.  picks > 0: y [*, W] holds expert rows, slot_of / pick_w [rows, picks].  extra [rows, W] joins y.  With plus_one
// the weights are stored around zero; store = 0 leaves x (and the history) as it is.  extras (null = none): see host_api.h.
extern "C" int atlas_add_normed(float* x, long long ldx, const void* y, long long ldy, const int* slot_of, const float* pick_w, int picks,
                                const void* extra, long long lde, const float* w, const float* out_w, const float* step, void* out,
                                long long ldo, int rows, int W, int plus_one, int store, int first, float eps, float scale, int f32,
                                const AtlasNormedExtras* extras, void* stream) {
  if (rows <= 0) return 0;
  if (W < 1 || W > 32768 || picks < 0 || (picks > 0 && (!slot_of || !pick_w)) || (first && w)) return -1;
  const AtlasNormedExtras o = extras ? *extras : AtlasNormedExtras{};
  if (o.hist && (o.hist_ld < (long long)rows * W || o.hist_index < 0)) return -3;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? add_normed<float>(x, ldx, y, ldy, slot_of, pick_w, picks, extra, lde, w, out_w, step, out, ldo, rows, W, plus_one, store, first, eps,
                                 scale, o, st)
             : add_normed<__nv_bfloat16>(x, ldx, y, ldy, slot_of, pick_w, picks, extra, lde, w, out_w, step, out, ldo, rows, W, plus_one, store,
                                         first, eps, scale, o, st);
}

// out [rows, N] = gelu_tanh(z) * table[ids[row], first + column] in the first n columns, 0 in the others
extern "C" int atlas_gelu_embedding(const void* z, long long ldz, const void* table, long long ldt, const long long* ids, int first, int n, int N,
                                    void* out, long long ldo, int rows, int f32, void* stream) {
  if (rows <= 0 || N <= 0) return 0;
  if (n < 0 || n > N || first < 0 || first + n > ldt) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (f32) {
    const bool vec = n % 4 == 0 && N % 4 == 0 && first % 4 == 0 && vec_ok<float, 4>(z, ldz) && vec_ok<float, 4>(table, ldt) && vec_ok<float, 4>(out, ldo);
    return vec ? launch_gelu_embedding<float, 4>(z, ldz, table, ldt, ids, first, n, N, out, ldo, rows, st)
               : launch_gelu_embedding<float, 1>(z, ldz, table, ldt, ids, first, n, N, out, ldo, rows, st);
  }
  using B = __nv_bfloat16;
  const bool vec = n % 8 == 0 && N % 8 == 0 && first % 8 == 0 && vec_ok<B, 8>(z, ldz) && vec_ok<B, 8>(table, ldt) && vec_ok<B, 8>(out, ldo);
  return vec ? launch_gelu_embedding<B, 8>(z, ldz, table, ldt, ids, first, n, N, out, ldo, rows, st)
             : launch_gelu_embedding<B, 1>(z, ldz, table, ldt, ids, first, n, N, out, ldo, rows, st);
}

// x [rows, H, D] (row stride ldx) times sigmoid(g [rows, H]), in place
extern "C" int atlas_head_gate(void* x, long long ldx, const float* g, long long ldg, int rows, int H, int D, int f32, void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (f32) return D % 4 == 0 && vec_ok<float, 4>(x, ldx) ? launch_head_gate<float, 4>(x, ldx, g, ldg, rows, H, D, st)
                                                         : launch_head_gate<float, 1>(x, ldx, g, ldg, rows, H, D, st);
  using B = __nv_bfloat16;
  return D % 8 == 0 && vec_ok<B, 8>(x, ldx) ? launch_head_gate<B, 8>(x, ldx, g, ldg, rows, H, D, st) : launch_head_gate<B, 1>(x, ldx, g, ldg, rows, H, D, st);
}
