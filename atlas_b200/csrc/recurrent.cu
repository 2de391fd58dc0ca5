// Linear recurrences with a diagonal decay on an fp32 state per head, varlen over the step's sequences:
//
//   Mamba-2 (SSD)   dt = max(softplus(dt_raw + dt_bias), dt_min),  a = exp(-exp(A_log) * dt)
//                   S[p][n] = a * S[p][n] + dt * x[p] * B[n];   y[p] = sum_n S[p][n] * C[n] + D * x[p]
//   WKV             w[n] = exp(-exp(raw[n] + w0[n]))
//                   y[p] = sum_n r[n] * (S[p][n] + u[n] * k[n] * v[p]);   S[p][n] = w[n] * S[p][n] + k[n] * v[p]
//
//   linear_scan_kernel   one CTA per (head, block of columns p, sequence).  KS lanes share a column; each holds NK state
//                        entries of CPT columns in registers (entry j*4+e of lane s is n = (j * KS + s) * 4 + e).  Four warps walk the rows
//                        while four more load the next kScanRows rows from global memory and turn them into the fp32
//                        coefficients (softplus, exponentials, row constants) in the other half of a double buffer.
//   linear_step_kernel   the same for one row per sequence (decode): no staging of rows, the state streams through.
//   Both serve speculative verify (no commit), the write-on-accept fold (row limit) and prefix-cache snapshots, like the
//   Gated-DeltaNet kernels (gdn.cu).  WKV's other piece of state, the previous token's input row, is stored here as well.
//   group_norm_gate_kernel   rms norm over channel groups joined with a SiLU gate: norm(y * silu(z)) * w (Mamba-2) or
//                        norm(y) * w * silu(z) (WKV)
//   conv1d_kernel        causal depth-wise convolution + bias + SiLU, window state of the last W - 1 inputs per channel
//
// Activations are bf16 or fp32 (template parameter T); states, decays and step sizes are fp32.
// Reference ops replaced: kernels/gb10/common/mamba2_ssm_decode.cu, mamba2_ssd_chunk.cu, causal_conv1d.cu, gated_rms_norm.
#include "common.cuh"
#include "host_api.h"
#include "vec_io.cuh"

namespace atlas {

enum { kMamba = 0, kWkv = 1 };

template <typename T>
struct ScanParams {
  // Mamba-2: rows [x | B | C] (a) and raw dt (b).  WKV: r, k, v and raw decay rows (a, b, c, d); a may be null (state only).
  const T* a; long long lda;
  const T* b; long long ldb;
  const T* c; long long ldc;
  const T* d; long long ldd;
  const float* A_log; const float* D; const float* dt_bias; float dt_min;
  const float* w0; const float* u;             // [H * N], [H, N]
  float* h;                                    // [slots, H, P, N]
  T* out; long long ldo;                       // [T, H * P]
  // WKV: previous-token rows x [T, W] -> shift [slots, W]
  const T* x; long long ldx; T* shift; int W;
  const int* query_start_loc; const int* state_slots; const unsigned char* has_state; const int* limit;
  const int* snap_rows; const int* snap_slots; int num_snaps_per_seq;
  int H, P, N, G, commit;
};

constexpr int kScanRows = 16, kGroup = 4;

ATLAS_DEVICE float softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }

// one head's coefficients of one row, element n (or column p)
template <typename T, int MODE>
ATLAS_DEVICE void row_key(const ScanParams<T>& p, int head, long long t, int n, float dtv, float* k, float* q, float* w) {
  if (n >= p.N) { *k = 0.f; *q = 0.f; *w = 0.f; return; }
  if (MODE == kMamba) {
    const T* row = p.a + t * p.lda + p.H * p.P + (head / (p.H / p.G)) * p.N;
    *k = dtv * to_f32(row[n]);
    *q = to_f32(row[p.G * p.N + n]);
    *w = 0.f;
  } else {
    const int i = head * p.N + n;
    *k = to_f32(p.b[t * p.ldb + i]);
    *q = p.a ? to_f32(p.a[t * p.lda + i]) : 0.f;
    *w = expf(-expf(to_f32(p.d[t * p.ldd + i]) + p.w0[i]));
  }
}
template <typename T, int MODE>
ATLAS_DEVICE float row_col(const ScanParams<T>& p, int head, long long t, int col) {
  if (col >= p.P) return 0.f;
  return MODE == kMamba ? to_f32(p.a[t * p.lda + head * p.P + col]) : to_f32(p.c[t * p.ldc + head * p.P + col]);
}

// One row's raw inputs as a warp holds them: element n = lane + 32 i of the keys, column lane + 32 i of the values.  The
// loads are unconditional (indices are clamped into the row, what lies outside is dropped when the row is used), so that all
// of them are in flight together.
template <typename T, int NI, int CI>
struct RowIn {
  T k[NI], q[NI], w[NI], x[CI], dt;
};
template <typename T, int MODE, int NI, int CI>
ATLAS_DEVICE void load_row(const ScanParams<T>& p, int head, long long t, int col0, int lane, RowIn<T, NI, CI>& in) {
  const T* qrow = MODE == kMamba ? p.a + t * p.lda + p.H * p.P + (p.G + head / (p.H / p.G)) * p.N
                                 : (p.a ? p.a + t * p.lda : p.b + t * p.ldb) + head * p.N;
  const T* krow = MODE == kMamba ? qrow - p.G * p.N : p.b + t * p.ldb + head * p.N;
  const T* wrow = MODE == kMamba ? krow : p.d + t * p.ldd + head * p.N;
  const T* xrow = (MODE == kMamba ? p.a + t * p.lda : p.c + t * p.ldc) + head * p.P;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = min(lane + 32 * i, p.N - 1);
    in.k[i] = krow[n];
    in.q[i] = qrow[n];
    if (MODE == kWkv) in.w[i] = wrow[n];
  }
#pragma unroll
  for (int i = 0; i < CI; ++i) in.x[i] = xrow[min(col0 + lane + 32 * i, p.P - 1)];
  if (MODE == kMamba) in.dt = p.b[t * p.ldb + head];
}

// WKV: rows of `x` that become a slot's previous-token row; the head CTAs share the W channels
template <typename T>
ATLAS_DEVICE void store_shift(const ScanParams<T>& p, int head, long long row, long long slot, int tid, int threads) {
  const int lo = (int)((long long)head * p.W / p.H), hi = (int)((long long)(head + 1) * p.W / p.H);
  for (int i = lo + tid; i < hi; i += threads) p.shift[slot * p.W + i] = p.x[row * p.ldx + i];
}

template <typename T, int MODE, int NK, int KS, int CPT>
__global__ void __launch_bounds__(256)
linear_scan_kernel(const ScanParams<T> p) {
  constexpr int NP = NK * KS, CL = 128 / KS, CB = CL * CPT;     // lanes' columns: c0 + i * CL
  constexpr int kRowF = NP * (MODE == kWkv ? 3 : 2) + CB;       // key, query (, decay) and column values of a row
  constexpr int NI = (NP + 31) / 32, CI = (CB + 31) / 32;
  extern __shared__ float sm[];                                 // [2][kScanRows][kRowF] then [2][kScanRows] row scalars
  float* scal = sm + 2 * kScanRows * kRowF;
  const int head = blockIdx.x, bseq = blockIdx.z;
  const int q0 = p.query_start_loc[bseq];
  const int qlen = p.query_start_loc[bseq + 1] - q0;
  const int n_rows = p.limit ? min(p.limit[bseq], qlen) : qlen;
  if (n_rows <= 0) return;
  const long long slot = p.state_slots[bseq];
  const bool walker = threadIdx.x < 128;
  const int tid = threadIdx.x & 127, warp = tid >> 5, lane = tid & 31;
  const int c0 = blockIdx.y * CB + tid / KS, s = tid % KS;
  const float neg_a = MODE == kMamba ? -expf(p.A_log[head]) : 0.f;
  const float dskip = MODE == kMamba ? p.D[head] : 0.f;
  const float dtb = MODE == kMamba ? p.dt_bias[head] : 0.f;

  float w0[MODE == kWkv ? NI : 1], un[MODE == kWkv ? NI : 1];
  if (MODE == kWkv) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int n = lane + 32 * i;
      w0[i] = n < p.N ? p.w0[head * p.N + n] : 0.f;
      un[i] = n < p.N ? p.u[head * p.N + n] : 0.f;
    }
  }
  // Loader warps: warp w owns rows w, w + 4, .. of every kScanRows-row block.  Their raw values are fetched one block before
  // they are turned into coefficients, so a whole block's time hides the memory latency.
  RowIn<T, NI, CI> in[kScanRows / 4];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int d = 0; d < kScanRows / 4; ++d)
      load_row<T, MODE, NI, CI>(p, head, q0 + min(r0 + warp + 4 * d, n_rows - 1), blockIdx.y * CB, lane, in[d]);
  };
  auto fill = [&](int buf, int r0) {
#pragma unroll
    for (int d = 0; d < kScanRows / 4; ++d) {
      if (r0 + warp + 4 * d >= n_rows) break;
      float* row = sm + (buf * kScanRows + warp + 4 * d) * kRowF;
      float sc = 0.f, dtv = 1.f;
      if (MODE == kMamba) {
        dtv = fmaxf(softplus(to_f32(in[d].dt) + dtb), p.dt_min);
        sc = expf(neg_a * dtv);
      }
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int n = lane + 32 * i;
        if (NP % 32 != 0 && n >= NP) break;
        const bool in_row = n < p.N;
        const float k = in_row ? to_f32(in[d].k[i]) : 0.f, q = in_row && (MODE == kMamba || p.a) ? to_f32(in[d].q[i]) : 0.f;
        row[n] = k * dtv;
        row[NP + n] = q;
        if (MODE == kWkv) {
          row[2 * NP + n] = in_row ? expf(-expf(to_f32(in[d].w[i]) + w0[i])) : 0.f;
          sc += q * un[i] * k;                                   // the bonus term's weight on v, the same for every column
        }
      }
#pragma unroll
      for (int i = 0; i < CI; ++i)
        if (lane + 32 * i < CB) row[kRowF - CB + lane + 32 * i] = to_f32(in[d].x[i]);
      if (MODE == kWkv) sc = warp_sum(sc);
      if (lane == 0) scal[buf * kScanRows + warp + 4 * d] = sc;
    }
  };

  float h[CPT][NK];
  auto each = [&](long long slot_of, auto fn) {                 // this thread's live state entries and their addresses
    if (!walker) return;
#pragma unroll
    for (int i = 0; i < CPT; ++i) {
      const int col = c0 + i * CL;
      if (col >= p.P) break;
      float* base = p.h + ((slot_of * p.H + head) * p.P + col) * p.N;
#pragma unroll
      for (int j = 0; j < NK / 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int n = (j * KS + s) * 4 + e;
          if (n < p.N) fn(h[i][j * 4 + e], base[n]);
        }
    }
  };
#pragma unroll
  for (int i = 0; i < CPT; ++i)
#pragma unroll
    for (int j = 0; j < NK; ++j) h[i][j] = 0.f;
  if (p.has_state[bseq]) each(slot, [](float& reg, float& mem) { reg = mem; });

  if (!walker) {
    fetch(0);
    fill(0, 0);
    fetch(kScanRows);
  }
  __syncthreads();
  for (int r0 = 0, buf = 0; r0 < n_rows; r0 += kScanRows, buf ^= 1) {
    if (!walker) {
      fill(buf ^ 1, r0 + kScanRows);
      fetch(r0 + 2 * kScanRows);
    } else {
      // rows in groups of kGroup: the sums over the lanes of a column are formed for a whole group together
      const int m = min(kScanRows, n_rows - r0);
      for (int rg = 0; rg < m; rg += kGroup) {
        float acc[kGroup][CPT], skip[kGroup][CPT];
#pragma unroll
        for (int g = 0; g < kGroup; ++g) {
          const int r = rg + g;
          if (r >= m) break;
          const float* row = sm + (buf * kScanRows + r) * kRowF;
          const float sc = scal[buf * kScanRows + r];
          float xv[CPT], part[CPT][4];
#pragma unroll
          for (int i = 0; i < CPT; ++i) {
            xv[i] = row[kRowF - CB + tid / KS + i * CL];
            skip[g][i] = (MODE == kMamba ? dskip : sc) * xv[i];
#pragma unroll
            for (int e = 0; e < 4; ++e) part[i][e] = 0.f;
          }
#pragma unroll
          for (int j = 0; j < NK / 4; ++j) {
            const float4 k4 = *reinterpret_cast<const float4*>(row + (j * KS + s) * 4);
            const float4 q4 = *reinterpret_cast<const float4*>(row + NP + (j * KS + s) * 4);
            const float k[4] = {k4.x, k4.y, k4.z, k4.w}, q[4] = {q4.x, q4.y, q4.z, q4.w};
            if constexpr (MODE == kMamba) {
#pragma unroll
              for (int i = 0; i < CPT; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                  h[i][j * 4 + e] = fmaf(h[i][j * 4 + e], sc, k[e] * xv[i]);
                  part[i][e] = fmaf(h[i][j * 4 + e], q[e], part[i][e]);
                }
            } else {
              const float4 w4 = *reinterpret_cast<const float4*>(row + 2 * NP + (j * KS + s) * 4);
              const float w[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
              for (int i = 0; i < CPT; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                  part[i][e] = fmaf(h[i][j * 4 + e], q[e], part[i][e]);
                  h[i][j * 4 + e] = fmaf(h[i][j * 4 + e], w[e], k[e] * xv[i]);
                }
            }
          }
#pragma unroll
          for (int i = 0; i < CPT; ++i) acc[g][i] = (part[i][0] + part[i][1]) + (part[i][2] + part[i][3]);
          for (int i = 0; i < p.num_snaps_per_seq; ++i)
            if (p.snap_rows[bseq * p.num_snaps_per_seq + i] == r0 + r + 1)
              each(p.snap_slots[bseq * p.num_snaps_per_seq + i], [](float& reg, float& mem) { mem = reg; });
        }
#pragma unroll
        for (int off = KS / 2; off > 0; off >>= 1)
#pragma unroll
          for (int g = 0; g < kGroup; ++g)
#pragma unroll
            for (int i = 0; i < CPT; ++i) acc[g][i] += __shfl_xor_sync(0xffffffffu, acc[g][i], off);
        if (s == 0 && p.out) {
#pragma unroll
          for (int g = 0; g < kGroup; ++g)
#pragma unroll
            for (int i = 0; i < CPT; ++i) {
              const int col = c0 + i * CL;
              if (rg + g < m && col < p.P)
                p.out[(long long)(q0 + r0 + rg + g) * p.ldo + head * p.P + col] = from_f32<T>(acc[g][i] + skip[g][i]);
            }
        }
      }
    }
    __syncthreads();
  }
  if (p.commit) each(slot, [](float& reg, float& mem) { mem = reg; });
  if (MODE == kWkv && blockIdx.y == 0) {
    for (int i = 0; i < p.num_snaps_per_seq; ++i) {
      const int r = p.snap_rows[bseq * p.num_snaps_per_seq + i];
      if (r > 0 && r <= n_rows) store_shift(p, head, q0 + r - 1, p.snap_slots[bseq * p.num_snaps_per_seq + i], threadIdx.x, 256);
    }
    if (p.commit) store_shift(p, head, q0 + n_rows - 1, slot, threadIdx.x, 256);
  }
}

// One row per sequence: grid (head, column blocks, sequence).  The row's coefficients are computed once per CTA, then every
// group of KS lanes streams the state rows of its columns (kCols of them, all loads in flight together).
constexpr int kStepCols = 4;
template <typename T, int MODE, int NK, int KS>
__global__ void __launch_bounds__(128)
linear_step_kernel(const ScanParams<T> p) {
  constexpr int NP = NK * KS, CB = 128 / KS * kStepCols;
  __shared__ __align__(16) float key[NP], qry[NP], dec[NP];
  __shared__ float part[4];
  chain_trigger();
  chain_wait();
  const int head = blockIdx.x, bseq = blockIdx.z;
  const long long t = p.query_start_loc[bseq];
  const long long slot = p.state_slots[bseq];
  const bool has = p.has_state[bseq] != 0;
  const int tid = threadIdx.x, s = tid % KS, c0 = blockIdx.y * CB + tid / KS;
  const bool full = p.N == NP;                                  // whole float4 pieces of the state
  float h[kStepCols][NK], xv[kStepCols];
#pragma unroll
  for (int i = 0; i < kStepCols; ++i) {
    const int col = c0 + i * (128 / KS);
    xv[i] = row_col<T, MODE>(p, head, t, col);
    const float* hs = p.h + (((long long)slot * p.H + head) * p.P + col) * p.N;
#pragma unroll
    for (int j = 0; j < NK / 4; ++j) {
      const int n = (j * KS + s) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (has && col < p.P) {
        if (full) {
          v = *reinterpret_cast<const float4*>(hs + n);
        } else {
          if (n < p.N) v.x = hs[n];
          if (n + 1 < p.N) v.y = hs[n + 1];
          if (n + 2 < p.N) v.z = hs[n + 2];
          if (n + 3 < p.N) v.w = hs[n + 3];
        }
      }
      h[i][j * 4] = v.x; h[i][j * 4 + 1] = v.y; h[i][j * 4 + 2] = v.z; h[i][j * 4 + 3] = v.w;
    }
  }
  float sc = 0.f, dtv = 0.f;
  if (MODE == kMamba) {
    dtv = fmaxf(softplus(to_f32(p.b[t * p.ldb + head]) + p.dt_bias[head]), p.dt_min);
    sc = expf(-expf(p.A_log[head]) * dtv);
  }
  for (int n = tid; n < NP; n += 128) {
    float k, q, w;
    row_key<T, MODE>(p, head, t, n, dtv, &k, &q, &w);
    key[n] = k; qry[n] = q; dec[n] = w;
    if (MODE == kWkv && n < p.N) sc += q * p.u[head * p.N + n] * k;
  }
  if (MODE == kWkv) {
    sc = warp_sum(sc);
    if ((tid & 31) == 0) part[tid >> 5] = sc;
  }
  __syncthreads();
  if (MODE == kWkv) sc = part[0] + part[1] + part[2] + part[3];
  const float skip = MODE == kMamba ? p.D[head] : sc;
#pragma unroll
  for (int i = 0; i < kStepCols; ++i) {
    const int col = c0 + i * (128 / KS);
    float acc = 0.f;
#pragma unroll
    for (int j = 0; j < NK / 4; ++j) {
      const float4 k4 = *reinterpret_cast<const float4*>(key + (j * KS + s) * 4);
      const float4 q4 = *reinterpret_cast<const float4*>(qry + (j * KS + s) * 4);
      const float k[4] = {k4.x, k4.y, k4.z, k4.w}, q[4] = {q4.x, q4.y, q4.z, q4.w};
      if constexpr (MODE == kMamba) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          h[i][j * 4 + e] = fmaf(h[i][j * 4 + e], sc, k[e] * xv[i]);
          acc = fmaf(h[i][j * 4 + e], q[e], acc);
        }
      } else {
        const float4 w4 = *reinterpret_cast<const float4*>(dec + (j * KS + s) * 4);
        const float w[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          acc = fmaf(h[i][j * 4 + e], q[e], acc);
          h[i][j * 4 + e] = fmaf(h[i][j * 4 + e], w[e], k[e] * xv[i]);
        }
      }
    }
#pragma unroll
    for (int off = KS / 2; off > 0; off >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, off);
    if (col >= p.P) continue;
    if (s == 0 && p.out) p.out[t * p.ldo + head * p.P + col] = from_f32<T>(fmaf(skip, xv[i], acc));
    if (p.commit) {
      float* hs = p.h + (((long long)slot * p.H + head) * p.P + col) * p.N;
#pragma unroll
      for (int j = 0; j < NK / 4; ++j) {
        const int n = (j * KS + s) * 4;
        if (full) {
          *reinterpret_cast<float4*>(hs + n) = make_float4(h[i][j * 4], h[i][j * 4 + 1], h[i][j * 4 + 2], h[i][j * 4 + 3]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (n + e < p.N) hs[n + e] = h[i][j * 4 + e];
        }
      }
    }
  }
  if (MODE == kWkv && p.commit && blockIdx.y == 0) store_shift(p, head, t, slot, tid, 128);
}

template <typename T, int MODE, int NK, int KS, int CPT>
static int launch_rows(const ScanParams<T>& p, int B, cudaStream_t st) {
  constexpr int CB = 128 / KS * CPT, NP = NK * KS;
  constexpr int smem = (2 * kScanRows * (NP * (MODE == kWkv ? 3 : 2) + CB) + 2 * kScanRows) * (int)sizeof(float);
  auto k = linear_scan_kernel<T, MODE, NK, KS, CPT>;
  if (smem > 40 * 1024 && ensure_dynamic_smem(reinterpret_cast<const void*>(k), smem) != cudaSuccess) return -20;
  k<<<dim3(p.H, (p.P + CB - 1) / CB, B), 256, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <typename T, int MODE, int NK, int KS>
static int launch_scan(const ScanParams<T>& p, int B, int one_row, cudaStream_t st) {
  if (one_row) {
    constexpr int CB = 128 / KS * kStepCols;
    launch_chain_if(true, linear_step_kernel<T, MODE, NK, KS>, dim3(p.H, (p.P + CB - 1) / CB, B), dim3(128), 0, st, p);
    return cudaGetLastError() == cudaSuccess ? 0 : -21;
  }
  // four columns per thread where that still gives most SMs a CTA: fewer shared-memory reads per state entry
  const long long lanes = (long long)p.H * B;
  if constexpr (KS >= 4) {                     // (fewer lanes per column already give a block of columns per CTA)
    if (lanes * ((p.P + 4 * (128 / KS) - 1) / (4 * (128 / KS))) >= 100) return launch_rows<T, MODE, NK, KS, 4>(p, B, st);
    if (lanes * ((p.P + 2 * (128 / KS) - 1) / (2 * (128 / KS))) >= 48) return launch_rows<T, MODE, NK, KS, 2>(p, B, st);
  }
  return launch_rows<T, MODE, NK, KS, 1>(p, B, st);
}

// `one_row`: every sequence of the step has exactly one row, no row limit and no snapshot
template <typename T, int MODE>
static int scan(const ScanParams<T>& p, int B, int one_row, cudaStream_t st) {
  if (B <= 0) return 0;
  if (p.H < 1 || p.P < 1 || p.N < 1 || (MODE == kMamba && (p.G < 1 || p.H % p.G))) return -1;
  if (one_row && (p.limit || p.num_snaps_per_seq)) return -3;
  if (p.N <= 8) return launch_scan<T, MODE, 8, 1>(p, B, one_row, st);
  if (p.N <= 16) return launch_scan<T, MODE, 8, 2>(p, B, one_row, st);
  if (p.N <= 32) return launch_scan<T, MODE, 8, 4>(p, B, one_row, st);
  if (p.N <= 64) return launch_scan<T, MODE, 16, 4>(p, B, one_row, st);
  if (p.N <= 128) return launch_scan<T, MODE, 16, 8>(p, B, one_row, st);
  if (p.N <= 256) return launch_scan<T, MODE, 16, 16>(p, B, one_row, st);
  return -2;
}

// ----------------------------------------------------------------------------- gated group norm
// TPG threads per (row, group): a quarter of a warp for head-sized groups, a warp, or a whole block for wide ones
template <typename T, int TPG, int V, bool kGateFirst>
__global__ void __launch_bounds__(256)
group_norm_gate_kernel(const T* __restrict__ y, long long ldy, const T* __restrict__ z, long long ldz,
                       const float* __restrict__ w, T* out, long long ldo, int rows, int groups, int gsize, float eps) {
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
  float ss = 0.f;
  for (int e = tid * V; e < gsize; e += TPG * V) {
    float f[V], g[V];
    load_vec<V>(yr + e, f);
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
  const float rstd = 1.f / sqrtf(ss / (float)gsize + eps);
  for (int e = tid * V; e < gsize; e += TPG * V) {
    float f[V], g[V], wv[V];
    load_vec<V>(yr + e, f);
    load_vec<V>(zr + e, g);
#pragma unroll
    for (int i = 0; i < V; ++i) wv[i] = w[g0 + e + i];
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = f[i] * rstd * wv[i] * (g[i] / (1.f + expf(-g[i])));
    store_vec<V>(out + t * ldo + g0 + e, f);
  }
}

template <typename T, int V, bool kGateFirst>
static int launch_gnorm(const void* y, long long ldy, const void* z, long long ldz, const float* w, void* out, long long ldo,
                        int rows, int groups, int gsize, float eps, cudaStream_t st) {
  const long long units = (long long)rows * groups;
  const T *yp = reinterpret_cast<const T*>(y), *zp = reinterpret_cast<const T*>(z);
  if (gsize >= 1024)
    launch_chain_if(rows <= 256, group_norm_gate_kernel<T, 256, V, kGateFirst>, dim3((unsigned)units), dim3(256), 0, st, yp, ldy, zp, ldz, w,
                    reinterpret_cast<T*>(out), ldo, rows, groups, gsize, eps);
  else if (gsize <= 128)
    launch_chain_if(rows <= 256, group_norm_gate_kernel<T, 8, V, kGateFirst>, dim3((unsigned)((units + 31) / 32)), dim3(256), 0, st, yp, ldy,
                    zp, ldz, w, reinterpret_cast<T*>(out), ldo, rows, groups, gsize, eps);
  else
    launch_chain_if(rows <= 256, group_norm_gate_kernel<T, 32, V, kGateFirst>, dim3((unsigned)((units + 7) / 8)), dim3(256), 0, st, yp, ldy,
                    zp, ldz, w, reinterpret_cast<T*>(out), ldo, rows, groups, gsize, eps);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <typename T>
static int gnorm(const void* y, long long ldy, const void* z, long long ldz, const float* w, void* out, long long ldo, int rows,
                 int groups, int gsize, float eps, int gate_first, cudaStream_t st) {
  if (sizeof(T) == 2 && gsize % 8 == 0 && (gsize < 1024 || gsize >= 2048) && vec_ok<T, 8>(y, ldy) && vec_ok<T, 8>(z, ldz) && vec_ok<T, 8>(out, ldo))
    return gate_first ? launch_gnorm<T, 8, true>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, st)
                      : launch_gnorm<T, 8, false>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, st);
  const bool vec = gsize % 4 == 0 && vec_ok<T, 4>(y, ldy) && vec_ok<T, 4>(z, ldz) && vec_ok<T, 4>(out, ldo);
  if (vec) return gate_first ? launch_gnorm<T, 4, true>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, st)
                             : launch_gnorm<T, 4, false>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, st);
  return gate_first ? launch_gnorm<T, 1, true>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, st)
                    : launch_gnorm<T, 1, false>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, st);
}

// ----------------------------------------------------------------------------- short convolution
constexpr int kMaxTaps = 16;
constexpr int kConvRows = 8;                   // consecutive rows of one thread (kTaps > 0: the window stays in registers)

// kTaps: number of taps known at compile time (0 = p.W, at most kMaxTaps, inputs re-read per row)
template <typename T, int kTaps, int V>
__global__ void __launch_bounds__(256)
conv1d_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ w, const T* __restrict__ bias, int C, int W,
              const T* __restrict__ state, const int* __restrict__ seq_of_token, const int* __restrict__ query_start_loc,
              const int* __restrict__ state_slots, const unsigned char* __restrict__ has_state, T* y, long long ldy, int rows) {
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
  const int t0 = blockIdx.x * kConvRows, t1 = min(rows, t0 + kConvRows);
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
    float acc[V];
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
      for (int i = 0; i < kN - 1; ++i)
#pragma unroll
        for (int v = 0; v < V; ++v) win[i][v] = win[i + 1][v];
    } else {
      for (int i = 0; i < taps; ++i) {
        float f[V];
        input(q0, rel, taps - 1 - i, slot, live, f);
#pragma unroll
        for (int v = 0; v < V; ++v) acc[v] = fmaf(f[v], to_f32(w[(long long)(c + v) * taps + i]), acc[v]);
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) acc[v] = acc[v] / (1.f + expf(-acc[v]));
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

template <typename T, int kTaps>
static int launch_conv(const void* x, long long ldx, const void* w, const void* bias, int C, int W, const void* state,
                       const int* seq, const int* qsl, const int* slots, const unsigned char* has, void* y, long long ldy,
                       int rows, cudaStream_t st) {
  const T *xp = reinterpret_cast<const T*>(x), *wp = reinterpret_cast<const T*>(w), *bp = reinterpret_cast<const T*>(bias);
  const T* sp = reinterpret_cast<const T*>(state);
  T* yp = reinterpret_cast<T*>(y);
  const unsigned gx = (rows + kConvRows - 1) / kConvRows;
  if (kTaps > 0 && rows > 256 && C % 4 == 0 && vec_ok<T, 4>(x, ldx) && vec_ok<T, 4>(y, ldy))
    launch_chain_if(false, conv1d_kernel<T, kTaps, (kTaps > 0 ? 4 : 1)>, dim3(gx, (C + 1023) / 1024), dim3(256), 0, st, xp, ldx, wp, bp, C, W,
                    sp, seq, qsl, slots, has, yp, ldy, rows);
  else
    launch_chain_if(rows <= 256, conv1d_kernel<T, kTaps, 1>, dim3(gx, (C + 255) / 256), dim3(256), 0, st, xp, ldx, wp, bp, C, W, sp, seq, qsl,
                    slots, has, yp, ldy, rows);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <typename T>
static int conv(const void* x, long long ldx, const void* w, const void* bias, int C, int W, const void* state, const int* seq,
                const int* qsl, const int* slots, const unsigned char* has, void* y, long long ldy, int rows, cudaStream_t st) {
  switch (W) {
    case 2: return launch_conv<T, 2>(x, ldx, w, bias, C, W, state, seq, qsl, slots, has, y, ldy, rows, st);
    case 3: return launch_conv<T, 3>(x, ldx, w, bias, C, W, state, seq, qsl, slots, has, y, ldy, rows, st);
    case 4: return launch_conv<T, 4>(x, ldx, w, bias, C, W, state, seq, qsl, slots, has, y, ldy, rows, st);
    default: return launch_conv<T, 0>(x, ldx, w, bias, C, W, state, seq, qsl, slots, has, y, ldy, rows, st);
  }
}

template <typename T>
static void fill_batch(ScanParams<T>& p, float* h, void* out, long long ldo, const int* qsl, const int* slots,
                       const unsigned char* has, const int* limit, const int* snap_rows, const int* snap_slots, int snaps, int H,
                       int P, int N, int G, int commit) {
  p.h = h; p.out = reinterpret_cast<T*>(out); p.ldo = ldo; p.query_start_loc = qsl; p.state_slots = slots; p.has_state = has;
  p.limit = limit; p.snap_rows = snap_rows; p.snap_slots = snap_slots; p.num_snaps_per_seq = snaps;
  p.H = H; p.P = P; p.N = N; p.G = G; p.commit = commit;
}

template <typename T>
static int mamba2(const void* y, long long ldy, const void* dt, long long lddt, const float* A_log, const float* D,
                  const float* dt_bias, float dt_min, float* h, void* out, long long ldo, const int* qsl, const int* slots,
                  const unsigned char* has, const int* limit, const int* snap_rows, const int* snap_slots, int snaps, int B, int H,
                  int P, int N, int G, int commit, int one_row, cudaStream_t st) {
  ScanParams<T> p = {};
  p.a = reinterpret_cast<const T*>(y); p.lda = ldy; p.b = reinterpret_cast<const T*>(dt); p.ldb = lddt;
  p.A_log = A_log; p.D = D; p.dt_bias = dt_bias; p.dt_min = dt_min;
  fill_batch(p, h, out, ldo, qsl, slots, has, limit, snap_rows, snap_slots, snaps, H, P, N, G, commit);
  return scan<T, kMamba>(p, B, one_row, st);
}

template <typename T>
static int wkv(const void* r, long long ldr, const void* k, long long ldk, const void* v, long long ldv, const void* raw, long long ldw,
               const float* w0, const float* u, float* h, void* out, long long ldo, const void* x, long long ldx, void* shift, int W,
               const int* qsl, const int* slots, const unsigned char* has, const int* limit, const int* snap_rows,
               const int* snap_slots, int snaps, int B, int H, int D, int commit, int one_row, cudaStream_t st) {
  ScanParams<T> p = {};
  p.a = reinterpret_cast<const T*>(r); p.lda = ldr; p.b = reinterpret_cast<const T*>(k); p.ldb = ldk;
  p.c = reinterpret_cast<const T*>(v); p.ldc = ldv; p.d = reinterpret_cast<const T*>(raw); p.ldd = ldw;
  p.w0 = w0; p.u = u; p.x = reinterpret_cast<const T*>(x); p.ldx = ldx; p.shift = reinterpret_cast<T*>(shift); p.W = W;
  fill_batch(p, h, out, ldo, qsl, slots, has, limit, snap_rows, snap_slots, snaps, H, D, D, 1, commit);
  return scan<T, kWkv>(p, B, one_row, st);
}

}  // namespace atlas

using namespace atlas;
using bf16 = __nv_bfloat16;

extern "C" int atlas_mamba2_scan(const void* y, long long ldy, const void* dt, long long lddt, const float* A_log, const float* D,
                                 const float* dt_bias, float dt_min, float* h, void* out, long long ldo, const int* qsl,
                                 const int* slots, const unsigned char* has, const int* limit, const int* snap_rows,
                                 const int* snap_slots, int snaps, int B, int H, int P, int N, int G, int commit, int one_row, int f32,
                                 void* stream) {
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? mamba2<float>(y, ldy, dt, lddt, A_log, D, dt_bias, dt_min, h, out, ldo, qsl, slots, has, limit, snap_rows, snap_slots, snaps,
                             B, H, P, N, G, commit, one_row, st)
             : mamba2<bf16>(y, ldy, dt, lddt, A_log, D, dt_bias, dt_min, h, out, ldo, qsl, slots, has, limit, snap_rows, snap_slots, snaps,
                            B, H, P, N, G, commit, one_row, st);
}

// r may be null: the state is advanced and nothing is written to `out` (write-on-accept fold)
extern "C" int atlas_wkv_scan(const void* r, long long ldr, const void* k, long long ldk, const void* v, long long ldv, const void* raw,
                              long long ldw, const float* w0, const float* u, float* h, void* out, long long ldo, const void* x,
                              long long ldx, void* shift, int W, const int* qsl, const int* slots, const unsigned char* has,
                              const int* limit, const int* snap_rows, const int* snap_slots, int snaps, int B, int H, int D, int commit,
                              int one_row, int f32, void* stream) {
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? wkv<float>(r, ldr, k, ldk, v, ldv, raw, ldw, w0, u, h, out, ldo, x, ldx, shift, W, qsl, slots, has, limit, snap_rows,
                          snap_slots, snaps, B, H, D, commit, one_row, st)
             : wkv<bf16>(r, ldr, k, ldk, v, ldv, raw, ldw, w0, u, h, out, ldo, x, ldx, shift, W, qsl, slots, has, limit, snap_rows,
                         snap_slots, snaps, B, H, D, commit, one_row, st);
}

extern "C" int atlas_group_norm_gate(const void* y, long long ldy, const void* z, long long ldz, const float* w, void* out, long long ldo,
                                     int rows, int groups, int gsize, float eps, int gate_first, int f32, void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? gnorm<float>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, gate_first, st)
             : gnorm<bf16>(y, ldy, z, ldz, w, out, ldo, rows, groups, gsize, eps, gate_first, st);
}

// depth-wise causal convolution + bias (may be null) + SiLU of [rows, C]; state [slots, C, W - 1]
extern "C" int atlas_conv1d_bias_silu(const void* x, long long ldx, const void* w, const void* bias, int C, int W, const void* state,
                                      const int* seq_of_token, const int* qsl, const int* slots, const unsigned char* has, void* y,
                                      long long ldy, int rows, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (W < 1 || W > kMaxTaps) return -1;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? conv<float>(x, ldx, w, bias, C, W, state, seq_of_token, qsl, slots, has, y, ldy, rows, st)
             : conv<bf16>(x, ldx, w, bias, C, W, state, seq_of_token, qsl, slots, has, y, ldy, rows, st);
}

extern "C" int atlas_conv1d_state(const void* x, long long ldx, int C, int W, void* state, const int* qsl, const int* slots,
                                  const unsigned char* has, const int* limit, const int* snap_rows, const int* snap_slots, int snaps,
                                  int B, int f32, void* stream) {
  if (B <= 0 || W == 1) return 0;
  if (W < 1 || W > kMaxTaps) return -1;
  dim3 grid((C + 255) / 256, B);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (f32) launch_chain_if(true, conv1d_state_kernel<float>, grid, dim3(256), 0, st, reinterpret_cast<const float*>(x), ldx, C, W,
                           reinterpret_cast<float*>(state), qsl, slots, has, limit, snap_rows, snap_slots, snaps);
  else launch_chain_if(true, conv1d_state_kernel<bf16>, grid, dim3(256), 0, st, reinterpret_cast<const bf16*>(x), ldx, C, W,
                       reinterpret_cast<bf16*>(state), qsl, slots, has, limit, snap_rows, snap_slots, snaps);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}
