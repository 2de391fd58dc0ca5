// Causal depth-wise convolution over a few taps with a window state per sequence (in front of Mamba-2 and the RG-LRU, on the input of
// any mixer):
//
//   conv1d_kernel        convolution + bias, then SiLU, or + the input itself; with one row per sequence it can move the window on
//   conv1d_state_kernel  the window after a step: the last W - 1 inputs per channel
//
// Activations are bf16 or fp32 (template parameter T).
// Reference op replaced: kernels/gb10/common/causal_conv1d.cu.
#include "common.cuh"
#include "host_api.h"
#include "vec_io.cuh"

namespace atlas {

constexpr int kMaxTaps = 16;
constexpr int kConvRows = 8;                   // consecutive rows of one thread in large steps (kTaps > 0: the window stays in registers)

enum ConvAfter { kConvPlain = 0, kConvSilu = 1, kConvAddInput = 2 };

// kTaps: number of taps known at compile time (0 = p.W, at most kMaxTaps, inputs re-read per row).  advance (one row per sequence):
// every thread replaces the window of its channels by the one that ends with its row.  span: rows of a block.
template <typename T, int kTaps, int V>
__global__ void __launch_bounds__(256)
conv1d_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ w, const T* __restrict__ bias, int C, int W,
              T* state, const int* __restrict__ seq_of_token, const int* __restrict__ query_start_loc, const int* __restrict__ state_slots,
              const unsigned char* __restrict__ has_state, T* y, long long ldy, int rows, int after, int advance, int span) {
  chain_trigger();
  chain_wait();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  const int taps = kTaps > 0 ? kTaps : W;
  constexpr int kN = kTaps > 0 ? kTaps : 1;
  float wt[kN][V], win[kN][V], bs[V];          // win[i]: the input i - (taps - 1) rows back
#pragma unroll
  for (int v = 0; v < V; ++v) {
    bs[v] = bias ? to_f32(bias[c + v]) : 0.f;
    if (kTaps > 0)
#pragma unroll
      for (int i = 0; i < kN; ++i) wt[i][v] = to_f32(w[(long long)(c + v) * taps + i]);
  }
  // input `back` rows before row `rel` of the chunk that starts at q0
  auto input = [&](int q0, int rel, int back, long long slot, bool live, float (&f)[V]) {
    if (back <= rel) {
      load_vec<V>(x + (long long)(q0 + rel - back) * ldx + c, f);
    } else {
#pragma unroll
      for (int v = 0; v < V; ++v)
        f[v] = live ? to_f32(state[(slot * C + c + v) * (taps - 1) + (taps - 1) - (back - rel)]) : 0.f;
    }
  };
  const int t0 = blockIdx.x * span, t1 = min(rows, t0 + span);
  if constexpr (kTaps > 0 && V > 1) {
    // all rows inside one portion, the window too: every load in flight at once
    const int b = seq_of_token[t0];
    if (t1 - t0 == kConvRows && seq_of_token[t1 - 1] == b && t0 - query_start_loc[b] >= kN - 1) {
      float in[kN - 1 + kConvRows][V];
#pragma unroll
      for (int r = 0; r < kN - 1 + kConvRows; ++r) load_vec<V>(x + (long long)(t0 - (kN - 1) + r) * ldx + c, in[r]);
#pragma unroll
      for (int r = 0; r < kConvRows; ++r) {
        float acc[V];
#pragma unroll
        for (int v = 0; v < V; ++v) {
          acc[v] = bs[v];
#pragma unroll
          for (int i = 0; i < kN; ++i) acc[v] = fmaf(in[r + i][v], wt[i][v], acc[v]);
          acc[v] = after == kConvSilu ? acc[v] * sigmoid_for<T>(acc[v]) : (after == kConvAddInput ? acc[v] + in[r + kN - 1][v] : acc[v]);
        }
        store_vec<V>(y + (long long)(t0 + r) * ldy + c, acc);
      }
      return;
    }
  }
  int seq = -1, q0 = 0;
  long long slot = 0;
  bool live = false;
  for (int t = t0; t < t1; ++t) {
    const int b = seq_of_token[t];
    const bool fresh = b != seq;
    if (fresh) {
      seq = b; q0 = query_start_loc[b]; slot = state_slots[b]; live = has_state[b] != 0;
    }
    const int rel = t - q0;
    float acc[V], own[V];
#pragma unroll
    for (int v = 0; v < V; ++v) acc[v] = bs[v];
    if constexpr (kTaps > 0) {
      if (fresh) {
#pragma unroll
        for (int i = 0; i < kN - 1; ++i) input(q0, rel, kN - 1 - i, slot, live, win[i]);
      }
      input(q0, rel, 0, slot, live, win[kN - 1]);
#pragma unroll
      for (int i = 0; i < kN; ++i)
#pragma unroll
        for (int v = 0; v < V; ++v) acc[v] = fmaf(win[i][v], wt[i][v], acc[v]);
#pragma unroll
      for (int v = 0; v < V; ++v) own[v] = win[kN - 1][v];
#pragma unroll
      for (int i = 0; i < kN - 1; ++i)
#pragma unroll
        for (int v = 0; v < V; ++v) win[i][v] = win[i + 1][v];
      if (advance) {
#pragma unroll
        for (int v = 0; v < V; ++v)
#pragma unroll
          for (int i = 0; i < kN - 1; ++i) state[(slot * C + c + v) * (kN - 1) + i] = from_f32<T>(win[i][v]);
      }
    } else {
      for (int i = 0; i < taps; ++i) {
        float f[V];
        input(q0, rel, taps - 1 - i, slot, live, f);
#pragma unroll
        for (int v = 0; v < V; ++v) {
          acc[v] = fmaf(f[v], to_f32(w[(long long)(c + v) * taps + i]), acc[v]);
          own[v] = f[v];                       // the last one is the row's own input
        }
      }
      if (advance) {
        for (int v = 0; v < V; ++v) {
          T* win0 = state + (slot * C + c + v) * (taps - 1);
          for (int i = 0; i < taps - 1; ++i) win0[i] = i + 1 < taps - 1 ? (live ? win0[i + 1] : from_f32<T>(0.f)) : from_f32<T>(own[v]);
        }
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) acc[v] = after == kConvSilu ? acc[v] / (1.f + expf(-acc[v])) : (after == kConvAddInput ? acc[v] + own[v] : acc[v]);
    store_vec<V>(y + (long long)t * ldy + c, acc);
  }
}

// new window = last W - 1 entries of (old window ++ first n rows of the chunk), n = limit ? limit[b] : q_len
template <typename T>
__global__ void __launch_bounds__(256)
conv1d_state_kernel(const T* __restrict__ x, long long ldx, int C, int W, T* state, const int* __restrict__ query_start_loc,
                    const int* __restrict__ state_slots, const unsigned char* __restrict__ has_state,
                    const int* __restrict__ limit, const int* __restrict__ snap_rows, const int* __restrict__ snap_slots,
                    int num_snaps_per_seq) {
  chain_trigger();
  chain_wait();
  const int b = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int q0 = query_start_loc[b];
  const int qlen = query_start_loc[b + 1] - q0;
  const long long slot = state_slots[b];
  const bool live = has_state[b] != 0;
  T old[kMaxTaps];
  for (int i = 0; i < W - 1; ++i) old[i] = live ? state[(slot * C + c) * (W - 1) + i] : from_f32<T>(0.f);
  auto window_after = [&](int n, long long dst) {
    for (int i = 0; i < W - 1; ++i) {
      const int src = n - (W - 1) + i;         // index into the chunk rows; negative -> old window
      state[(dst * C + c) * (W - 1) + i] = src >= 0 ? x[(long long)(q0 + src) * ldx + c] : old[(W - 1) + src];
    }
  };
  for (int s = 0; s < num_snaps_per_seq; ++s) {
    const int n = snap_rows[b * num_snaps_per_seq + s];
    if (n > 0 && n <= qlen) window_after(n, snap_slots[b * num_snaps_per_seq + s]);
  }
  const int n = limit ? limit[b] : qlen;
  if (n > 0) window_after(n, slot);
}

// the same for bf16 windows of three inputs, eight channels per thread
__global__ void __launch_bounds__(128)
conv1d_state4_kernel(const __nv_bfloat16* __restrict__ x, long long ldx, int C, __nv_bfloat16* state, const int* __restrict__ query_start_loc,
                     const int* __restrict__ state_slots, const unsigned char* __restrict__ has_state, const int* __restrict__ limit,
                     const int* __restrict__ snap_rows, const int* __restrict__ snap_slots, int num_snaps_per_seq) {
  chain_trigger();
  chain_wait();
  const int b = blockIdx.y, c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= C) return;
  const int q0 = query_start_loc[b], qlen = query_start_loc[b + 1] - q0;
  const long long slot = state_slots[b];
  union Window { uint4 v[3]; __nv_bfloat16 e[8][3]; };
  union Row { uint4 v; __nv_bfloat16 e[8]; };
  Window old;
#pragma unroll
  for (int i = 0; i < 3; ++i)
    old.v[i] = has_state[b] ? reinterpret_cast<const uint4*>(state + (slot * C + c) * 3)[i] : make_uint4(0u, 0u, 0u, 0u);
  auto window_after = [&](int n, long long dst) {
    Row r[3];
#pragma unroll
    for (int i = 0; i < 3; ++i) {
      const int src = n - 3 + i;
      r[i].v = src >= 0 ? *reinterpret_cast<const uint4*>(x + (long long)(q0 + src) * ldx + c) : make_uint4(0u, 0u, 0u, 0u);
    }
    Window w;
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      w.e[k][0] = n >= 3 ? r[0].e[k] : (n == 2 ? old.e[k][2] : old.e[k][1]);
      w.e[k][1] = n >= 2 ? r[1].e[k] : old.e[k][2];
      w.e[k][2] = r[2].e[k];
    }
#pragma unroll
    for (int i = 0; i < 3; ++i) reinterpret_cast<uint4*>(state + (dst * C + c) * 3)[i] = w.v[i];
  };
  for (int s = 0; s < num_snaps_per_seq; ++s) {
    const int n = snap_rows[b * num_snaps_per_seq + s];
    if (n > 0 && n <= qlen) window_after(n, snap_slots[b * num_snaps_per_seq + s]);
  }
  const int n = limit ? limit[b] : qlen;
  if (n > 0) window_after(n, slot);
}

template <typename T, int kTaps>
static int launch_conv(const void* x, long long ldx, const void* w, const void* bias, int C, int W, void* state,
                       const int* seq, const int* qsl, const int* slots, const unsigned char* has, void* y, long long ldy,
                       int rows, int after, int advance, cudaStream_t st) {
  const T *xp = reinterpret_cast<const T*>(x), *wp = reinterpret_cast<const T*>(w), *bp = reinterpret_cast<const T*>(bias);
  T* sp = reinterpret_cast<T*>(state);
  T* yp = reinterpret_cast<T*>(y);
  const int span = rows <= 256 ? 1 : kConvRows;
  const unsigned gx = (rows + span - 1) / span;
  if (kTaps > 0 && rows > 256 && C % 4 == 0 && vec_ok<T, 4>(x, ldx) && vec_ok<T, 4>(y, ldy))
    launch_chain_if(false, conv1d_kernel<T, kTaps, (kTaps > 0 ? 4 : 1)>, dim3(gx, (C + 1023) / 1024), dim3(256), 0, st, xp, ldx, wp, bp, C, W,
                    sp, seq, qsl, slots, has, yp, ldy, rows, after, advance, span);
  else
    launch_chain_if(rows <= 256, conv1d_kernel<T, kTaps, 1>, dim3(gx, (C + 255) / 256), dim3(256), 0, st, xp, ldx, wp, bp, C, W, sp, seq, qsl,
                    slots, has, yp, ldy, rows, after, advance, span);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <typename T>
static int conv(const void* x, long long ldx, const void* w, const void* bias, int C, int W, void* state, const int* seq, const int* qsl,
                const int* slots, const unsigned char* has, void* y, long long ldy, int rows, int after, int advance, cudaStream_t st) {
  switch (W) {
    case 1: return launch_conv<T, 1>(x, ldx, w, bias, C, W, state, seq, qsl, slots, has, y, ldy, rows, after, advance, st);
    case 2: return launch_conv<T, 2>(x, ldx, w, bias, C, W, state, seq, qsl, slots, has, y, ldy, rows, after, advance, st);
    case 3: return launch_conv<T, 3>(x, ldx, w, bias, C, W, state, seq, qsl, slots, has, y, ldy, rows, after, advance, st);
    case 4: return launch_conv<T, 4>(x, ldx, w, bias, C, W, state, seq, qsl, slots, has, y, ldy, rows, after, advance, st);
    default: return launch_conv<T, 0>(x, ldx, w, bias, C, W, state, seq, qsl, slots, has, y, ldy, rows, after, advance, st);
  }
}

}  // namespace atlas

using namespace atlas;
using bf16 = __nv_bfloat16;

// depth-wise causal convolution + bias (may be null), then SiLU where `silu` says so, of [rows, C]; state [slots, C, W - 1]
extern "C" int atlas_conv1d_bias_silu(const void* x, long long ldx, const void* w, const void* bias, int C, int W, const void* state,
                                      const int* seq_of_token, const int* qsl, const int* slots, const unsigned char* has, void* y,
                                      long long ldy, int rows, int silu, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (W < 1 || W > kMaxTaps) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const int after = silu ? kConvSilu : kConvPlain;
  return f32 ? conv<float>(x, ldx, w, bias, C, W, const_cast<void*>(state), seq_of_token, qsl, slots, has, y, ldy, rows, after, 0, st)
             : conv<bf16>(x, ldx, w, bias, C, W, const_cast<void*>(state), seq_of_token, qsl, slots, has, y, ldy, rows, after, 0, st);
}

// y = x + convolution of x; advance (steps of one row per sequence): the windows move on in the same launch
extern "C" int atlas_conv1d_add(const void* x, long long ldx, const void* w, int C, int W, void* state, const int* seq_of_token, const int* qsl,
                                const int* slots, const unsigned char* has, void* y, long long ldy, int rows, int advance, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (W < 1 || W > kMaxTaps) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? conv<float>(x, ldx, w, nullptr, C, W, state, seq_of_token, qsl, slots, has, y, ldy, rows, kConvAddInput, advance, st)
             : conv<bf16>(x, ldx, w, nullptr, C, W, state, seq_of_token, qsl, slots, has, y, ldy, rows, kConvAddInput, advance, st);
}

extern "C" int atlas_conv1d_state(const void* x, long long ldx, int C, int W, void* state, const int* qsl, const int* slots,
                                  const unsigned char* has, const int* limit, const int* snap_rows, const int* snap_slots, int snaps,
                                  int B, int f32, void* stream) {
  if (B <= 0 || W == 1) return 0;
  if (W < 1 || W > kMaxTaps) return -1;
  dim3 grid((C + 255) / 256, B);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (!f32 && W == 4 && C % 8 == 0 && vec_ok<bf16, 8>(x, ldx) && vec_ok<bf16, 8>(state, 0)) {
    launch_chain_if(true, conv1d_state4_kernel, dim3((C / 8 + 127) / 128, B), dim3(128), 0, st, reinterpret_cast<const bf16*>(x), ldx, C,
                    reinterpret_cast<bf16*>(state), qsl, slots, has, limit, snap_rows, snap_slots, snaps);
    return cudaGetLastError() == cudaSuccess ? 0 : -21;
  }
  if (f32) launch_chain_if(true, conv1d_state_kernel<float>, grid, dim3(256), 0, st, reinterpret_cast<const float*>(x), ldx, C, W,
                           reinterpret_cast<float*>(state), qsl, slots, has, limit, snap_rows, snap_slots, snaps);
  else launch_chain_if(true, conv1d_state_kernel<bf16>, grid, dim3(256), 0, st, reinterpret_cast<const bf16*>(x), ldx, C, W,
                       reinterpret_cast<bf16*>(state), qsl, slots, has, limit, snap_rows, snap_slots, snaps);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}
