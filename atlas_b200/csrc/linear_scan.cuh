// Linear recurrences with a diagonal decay on an fp32 state per head, varlen over the step's sequences (templates; the entry
// points are in recurrent.cu and mlstm.cu):
//
//   Mamba-2 (SSD)   dt = max(softplus(dt_raw + dt_bias), dt_min),  a = exp(-exp(A_log) * dt)
//                   S[p][n] = a * S[p][n] + dt * x[p] * B[n];   y[p] = sum_n S[p][n] * C[n] + D * x[p]
//   WKV             w[n] = exp(-exp(raw[n] + w0[n]))
//                   y[p] = sum_n r[n] * (S[p][n] + u[n] * k[n] * v[p]);   S[p][n] = w[n] * S[p][n] + k[n] * v[p]
//
//   mLSTM           S[p][n] = e^la * S[p][n] + e^lb * k[n] * v[p];   y[p] = scale * sum_n q[n] * S[p][n], with the log factors
//                   la, lb of mlstm_gates_kernel (mlstm.cu) and one more value channel that is always 1 (the normaliser n)
//
//   linear_scan_kernel   one CTA per (head, block of columns p, sequence).  KS lanes share a column; each holds NK state
//                        entries of CPT columns in registers (entry j*4+e of lane s is n = (j * KS + s) * 4 + e).  Four warps walk the rows
//                        while four more load the next kScanRows rows from global memory and turn them into the fp32
//                        coefficients (softplus, exponentials, row constants) in the other half of a double buffer.
//   linear_step_kernel   the same for one row per sequence (decode): no staging of rows, the state streams through.
//   Both serve speculative verify (no commit), the write-on-accept fold (row limit) and prefix-cache snapshots, like the
//   Gated-DeltaNet kernels (gdn.cu).  WKV's other piece of state, the previous token's input row, is stored here as well.
//
// Activations are bf16 or fp32 (template parameter T); states, decays and step sizes are fp32.
// Reference ops replaced: kernels/gb10/common/mamba2_ssm_decode.cu, mamba2_ssd_chunk.cu.
#pragma once
#include "common.cuh"
#include "vec_io.cuh"

namespace atlas {

enum { kMamba = 0, kWkv = 1, kMlstm = 2 };

template <typename T>
struct ScanParams {
  // Mamba-2: rows [x | B | C] (a) and raw dt (b).  WKV: r, k, v and raw decay rows (a, b, c, d); a may be null (state only).
  // mLSTM: q, k, v rows (a, b, c; a may be null) and per row and head the log factors la, lb and the running maximum; P counts
  // the channel of the normaliser.
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
  // mLSTM: [T, H] each; den receives max(|n . q|, e^-top) + 1e-6
  const float* la; const float* lb; const float* top; float* den; float q_scale;
  const int* query_start_loc; const int* state_slots; const unsigned char* has_state; const int* limit;
  const int* snap_rows; const int* snap_slots; int num_snaps_per_seq;
  int H, P, N, G, commit;
};

constexpr int kScanRows = 16, kGroup = 4;
constexpr float kMlstmEps = 1e-6f;

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
    *k = to_f32(p.b[t * p.ldb + i]) * (MODE == kMlstm ? dtv : 1.f);
    *q = p.a ? to_f32(p.a[t * p.lda + i]) * (MODE == kMlstm ? p.q_scale : 1.f) : 0.f;
    *w = MODE == kMlstm ? 0.f : expf(-expf(to_f32(p.d[t * p.ldd + i]) + p.w0[i]));
  }
}
template <typename T, int MODE>
ATLAS_DEVICE float row_col(const ScanParams<T>& p, int head, long long t, int col) {
  if (col >= p.P) return 0.f;
  if (MODE == kMlstm) return col == p.P - 1 ? 1.f : to_f32(p.c[t * p.ldc + head * (p.P - 1) + col]);
  return MODE == kMamba ? to_f32(p.a[t * p.lda + head * p.P + col]) : to_f32(p.c[t * p.ldc + head * p.P + col]);
}

// One row's raw inputs as a warp holds them: element n = lane + 32 i of the keys, column lane + 32 i of the values.  The
// loads are unconditional (indices are clamped into the row, what lies outside is dropped when the row is used), so that all
// of them are in flight together.
template <typename T, int NI, int CI>
struct RowIn {
  T k[NI], q[NI], w[NI], x[CI], dt;
  float la, lb;
};
template <typename T, int MODE, int NI, int CI>
ATLAS_DEVICE void load_row(const ScanParams<T>& p, int head, long long t, int col0, int lane, RowIn<T, NI, CI>& in) {
  const T* qrow = MODE == kMamba ? p.a + t * p.lda + p.H * p.P + (p.G + head / (p.H / p.G)) * p.N
                                 : (p.a ? p.a + t * p.lda : p.b + t * p.ldb) + head * p.N;
  const T* krow = MODE == kMamba ? qrow - p.G * p.N : p.b + t * p.ldb + head * p.N;
  const T* wrow = MODE == kWkv ? p.d + t * p.ldd + head * p.N : krow;
  const int channels = MODE == kMlstm ? p.P - 1 : p.P;
  const T* xrow = (MODE == kMamba ? p.a + t * p.lda : p.c + t * p.ldc) + head * channels;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = min(lane + 32 * i, p.N - 1);
    in.k[i] = krow[n];
    in.q[i] = qrow[n];
    if (MODE == kWkv) in.w[i] = wrow[n];
  }
#pragma unroll
  for (int i = 0; i < CI; ++i) in.x[i] = xrow[min(col0 + lane + 32 * i, channels - 1)];
  if (MODE == kMamba) in.dt = p.b[t * p.ldb + head];
  if (MODE == kMlstm) {
    in.la = p.la[t * p.H + head];
    in.lb = p.lb[t * p.H + head];
  }
}

// WKV: rows of `x` that become a slot's previous-token row; the head CTAs share the W channels
template <typename T>
ATLAS_DEVICE void store_shift(const ScanParams<T>& p, int head, long long row, long long slot, int tid, int threads) {
  const int lo = (int)((long long)head * p.W / p.H), hi = (int)((long long)(head + 1) * p.W / p.H);
  for (int i = lo + tid; i < hi; i += threads) p.shift[slot * p.W + i] = p.x[row * p.ldx + i];
}

template <typename T, int MODE>
ATLAS_DEVICE void store_out(const ScanParams<T>& p, int head, long long t, int col, float y) {
  if (MODE != kMlstm) p.out[t * p.ldo + head * p.P + col] = from_f32<T>(y);
  else if (col < p.P - 1) p.out[t * p.ldo + head * (p.P - 1) + col] = from_f32<T>(y);
  else p.den[t * p.H + head] = fmaxf(fabsf(y), expf(-p.top[t * p.H + head])) + kMlstmEps;
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
      if (MODE == kMlstm) {
        dtv = expf(in[d].lb);
        sc = expf(in[d].la);
      }
      const float qs = MODE == kMlstm ? p.q_scale : 1.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int n = lane + 32 * i;
        if (NP % 32 != 0 && n >= NP) break;
        const bool in_row = n < p.N;
        const float k = in_row ? to_f32(in[d].k[i]) : 0.f, q = in_row && (MODE == kMamba || p.a) ? to_f32(in[d].q[i]) : 0.f;
        row[n] = k * dtv;
        row[NP + n] = q * qs;
        if (MODE == kWkv) {
          row[2 * NP + n] = in_row ? expf(-expf(to_f32(in[d].w[i]) + w0[i])) : 0.f;
          sc += q * un[i] * k;                                   // the bonus term's weight on v, the same for every column
        }
      }
#pragma unroll
      for (int i = 0; i < CI; ++i)
        if (lane + 32 * i < CB)
          row[kRowF - CB + lane + 32 * i] = MODE == kMlstm && blockIdx.y * CB + lane + 32 * i == p.P - 1 ? 1.f : to_f32(in[d].x[i]);
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
            skip[g][i] = MODE == kMlstm ? 0.f : (MODE == kMamba ? dskip : sc) * xv[i];
#pragma unroll
            for (int e = 0; e < 4; ++e) part[i][e] = 0.f;
          }
#pragma unroll
          for (int j = 0; j < NK / 4; ++j) {
            const float4 k4 = *reinterpret_cast<const float4*>(row + (j * KS + s) * 4);
            const float4 q4 = *reinterpret_cast<const float4*>(row + NP + (j * KS + s) * 4);
            const float k[4] = {k4.x, k4.y, k4.z, k4.w}, q[4] = {q4.x, q4.y, q4.z, q4.w};
            if constexpr (MODE != kWkv) {
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
              if (rg + g < m && col < p.P) store_out<T, MODE>(p, head, q0 + r0 + rg + g, col, acc[g][i] + skip[g][i]);
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
  if (MODE == kMlstm) {
    dtv = expf(p.lb[t * p.H + head]);
    sc = expf(p.la[t * p.H + head]);
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
  const float skip = MODE == kMlstm ? 0.f : (MODE == kMamba ? p.D[head] : sc);
#pragma unroll
  for (int i = 0; i < kStepCols; ++i) {
    const int col = c0 + i * (128 / KS);
    float acc = 0.f;
#pragma unroll
    for (int j = 0; j < NK / 4; ++j) {
      const float4 k4 = *reinterpret_cast<const float4*>(key + (j * KS + s) * 4);
      const float4 q4 = *reinterpret_cast<const float4*>(qry + (j * KS + s) * 4);
      const float k[4] = {k4.x, k4.y, k4.z, k4.w}, q[4] = {q4.x, q4.y, q4.z, q4.w};
      if constexpr (MODE != kWkv) {
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
    if (s == 0 && p.out) store_out<T, MODE>(p, head, t, col, fmaf(skip, xv[i], acc));
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
  if constexpr (MODE == kMlstm) {
    if (p.N <= 512) return launch_scan<T, MODE, 16, 32>(p, B, one_row, st);
  }
  return -2;
}

template <typename T>
static void fill_batch(ScanParams<T>& p, float* h, void* out, long long ldo, const int* qsl, const int* slots,
                       const unsigned char* has, const int* limit, const int* snap_rows, const int* snap_slots, int snaps, int H,
                       int P, int N, int G, int commit) {
  p.h = h; p.out = reinterpret_cast<T*>(out); p.ldo = ldo; p.query_start_loc = qsl; p.state_slots = slots; p.has_state = has;
  p.limit = limit; p.snap_rows = snap_rows; p.snap_slots = snap_slots; p.num_snaps_per_seq = snaps;
  p.H = H; p.P = P; p.N = N; p.G = G; p.commit = commit;
}

}  // namespace atlas
