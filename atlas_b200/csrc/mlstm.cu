// mLSTM matrix memory (xLSTM) on an fp32 state per head, varlen over the step's sequences.
//
//   i = cap tanh((i_raw + b_i) / cap),  f = logsigmoid(cap tanh((f_raw + b_f) / cap)),  m_t = max(f + m_(t-1), i)
//   S_t = e^la S_(t-1) + e^lb v k^T,  la = f + m_(t-1) - m_t <= 0,  lb = i - m_t <= 0;  n likewise with v = 1
//   num = scale S q,  den = max(|scale n . q|, e^-m) + 1e-6
//
//   mlstm_gates_kernel   one warp per (head, sequence): 32 rows a step; the running maximum is a prefix maximum of i - F with F
//                        the prefix sum of f.  Writes la, lb and m of every row and the slot's m.
//   linear_scan / linear_step (linear_scan.cuh)   the sequential form: fp32 activations, short portions, decode rows
//   mlstm_chunk_kernel   chunks of 64 rows on the tensor cores (bf16 activations).  One CTA per (head, 64 value channels,
//                        sequence) walks the chunks; S^T stays in the accumulator registers of four warps, 16 value channels
//                        each, for the whole sequence.  Per chunk, with cum the prefix sum of la:
//                          P[i][j] = scale q_i . k_j e^(cum_i - cum_j + lb_j)  (j <= i)
//                          num^T   = e^cum_i scale S^T Q^T + V^T P^T
//                          S^T     = e^cum_end S^T + (V e^(cum_end - cum_j + lb_j))^T K
//                        q, k and v are bf16 as they are; the fp32 operands (S, P, weighted V) enter as two bf16 terms each, so
//                        the products keep about 16 mantissa bits.
#include "common.cuh"
#include "host_api.h"
#include "linear_scan.cuh"
#include "mma_util.cuh"
#include "vec_io.cuh"

namespace atlas {

struct MlstmGateParams {
  const float* raw; long long ld;              // [T, 2 H]: input gates, forget gates
  const float* bias;                           // [2 H]
  float cap;
  float* m;                                    // [slots, H]
  float* la; float* lb; float* top;            // [T, H]
  const int* query_start_loc; const int* state_slots; const unsigned char* has_state; const int* limit;
  const int* snap_rows; const int* snap_slots; int snaps;
  int H, commit;
};

__global__ void __launch_bounds__(128)
mlstm_gates_kernel(const MlstmGateParams p) {
  chain_trigger();
  chain_wait();
  const int head = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31, b = blockIdx.y;
  if (head >= p.H) return;
  const int q0 = p.query_start_loc[b], qlen = p.query_start_loc[b + 1] - q0;
  const int n = p.limit ? min(p.limit[b], qlen) : qlen;
  if (n <= 0) return;
  const long long slot = p.state_slots[b];
  const float bi = p.bias[head], bf = p.bias[p.H + head];
  float m0 = p.has_state[b] ? p.m[slot * p.H + head] : 0.f;
  for (int r0 = 0; r0 < n; r0 += 32) {
    const int r = r0 + lane;
    const bool live = r < n;
    const long long t = q0 + min(r, n - 1);
    const float iv = p.cap * tanhf((p.raw[t * p.ld + head] + bi) / p.cap);
    const float z = p.cap * tanhf((p.raw[t * p.ld + p.H + head] + bf) / p.cap);
    const float fv = live ? fminf(z, 0.f) - log1pf(expf(-fabsf(z))) : 0.f;
    float F = fv;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, F, o);
      if (lane >= o) F += up;
    }
    float G = live ? iv - F : -INFINITY;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, G, o);
      if (lane >= o) G = fmaxf(G, up);
    }
    const float mr = F + fmaxf(m0, G);
    float prev = __shfl_up_sync(0xffffffffu, mr, 1);
    if (lane == 0) prev = m0;
    if (live) {
      p.la[t * p.H + head] = fminf(fv + prev - mr, 0.f);
      p.lb[t * p.H + head] = fminf(iv - mr, 0.f);
      p.top[t * p.H + head] = mr;
      for (int s = 0; s < p.snaps; ++s)
        if (p.snap_rows[b * p.snaps + s] == r + 1) p.m[(long long)p.snap_slots[b * p.snaps + s] * p.H + head] = mr;
      if (p.commit && r == n - 1) p.m[slot * p.H + head] = mr;
    }
    m0 = __shfl_sync(0xffffffffu, mr, 31);
  }
}

// ----------------------------------------------------------------------------- chunked form
constexpr int kMlRows = 64, kMlCols = 64;      // rows of a chunk, value channels of a CTA
constexpr int kMlPS = kMlRows + 8, kMlVS = kMlCols + 8;

struct MlstmChunkParams {
  const __nv_bfloat16* q; long long ldq;
  const __nv_bfloat16* k; long long ldk;
  const __nv_bfloat16* v; long long ldv;
  const float* la; const float* lb; const float* top;
  float scale;
  float* h;                                    // [slots, H, V + 1, D]
  __nv_bfloat16* out; long long ldo;           // [T, H * V]
  float* den;                                  // [T, H]
  const int* query_start_loc; const int* state_slots; const unsigned char* has_state;
  const int* snap_rows; const int* snap_slots; int snaps;
  int H, V, D, commit;
};

template <int DK>
struct MlstmSmem {
  static constexpr int kQS = DK + 8;           // padded row: ldmatrix phases hit distinct banks
  __nv_bfloat16 q[kMlRows * kQS];
  __nv_bfloat16 k[kMlRows * kQS];
  __nv_bfloat16 v[kMlRows * kMlVS];
  __nv_bfloat16 ph[kMlRows * kMlPS];
  __nv_bfloat16 pl[kMlRows * kMlPS];
  __nv_bfloat16 o[4][kMlRows * 24];            // a warp's 16 output channels per row, rows of 48 bytes
  float n[DK];
  float cum[kMlRows], lb[kMlRows], w[kMlRows], rowsum[kMlRows];
};

template <int DK>
__global__ void __launch_bounds__(128)
mlstm_chunk_kernel(const MlstmChunkParams p) {
  extern __shared__ __align__(16) uint8_t raw_smem[];
  using Sm = MlstmSmem<DK>;
  Sm& sm = *reinterpret_cast<Sm*>(raw_smem);
  constexpr int QS = Sm::kQS, KT = DK / 8;
  const int head = blockIdx.x, c0 = blockIdx.y * kMlCols, b = blockIdx.z;
  const int q0 = p.query_start_loc[b], n_rows = p.query_start_loc[b + 1] - q0;
  if (n_rows <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const long long slot = p.state_slots[b];
  const bool owner = blockIdx.y == 0;          // this CTA also keeps the normaliser and writes the denominators
  const int D = p.D, V = p.V;
  const int row_of = c0 + warp * 16 + g;       // this thread's value channels: row_of and row_of + 8

  float S[KT][4];
  auto each = [&](long long sl, auto fn) {     // this thread's live state entries and their addresses
    float* base = p.h + (sl * p.H + head) * (long long)(V + 1) * D;
#pragma unroll
    for (int j = 0; j < KT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = row_of + 8 * (e >> 1), c = j * 8 + 2 * t4 + (e & 1);
        if (r < V && c < D) fn(S[j][e], base[(long long)r * D + c]);
      }
  };
  auto save = [&](long long sl) {
    each(sl, [](float& reg, float& mem) { mem = reg; });
    if (owner)
      for (int c = tid; c < D; c += 128) p.h[((sl * p.H + head) * (long long)(V + 1) + V) * D + c] = sm.n[c];
  };
#pragma unroll
  for (int j = 0; j < KT; ++j) S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.f;
  for (int c = tid; c < DK; c += 128) sm.n[c] = 0.f;
  if (p.has_state[b]) {
    each(slot, [](float& reg, float& mem) { reg = mem; });
    if (owner)
      for (int c = tid; c < D; c += 128) sm.n[c] = p.h[((slot * p.H + head) * (long long)(V + 1) + V) * D + c];
  }

  const uint32_t aq = smem_u32(sm.q), ak = smem_u32(sm.k), av = smem_u32(sm.v), aph = smem_u32(sm.ph), apl = smem_u32(sm.pl);
  // ldmatrix lane addresses.  A / row-major [row][k]: lanes 0..15 rows, lane >> 4 the k half.  B from [n][k]: two n8 tiles, lanes
  // 0..7 / 16..23 rows of the tiles, bit 3 the k half.  Transposed: lanes 0..15 rows (k), lane >> 4 the column half.
  const int a_row = lane & 15, a_col = (lane >> 4) * 8;
  const int b_row = (lane & 7) + ((lane >> 4) << 3), b_col = ((lane >> 3) & 1) * 8;
  const float LOG2E = 1.4426950408889634f;

  for (int r0 = 0; r0 < n_rows;) {
    int r1 = min(r0 + kMlRows, n_rows);
    for (int s = 0; s < p.snaps; ++s) {        // a snapshot row ends a chunk early
      const int sr = p.snap_rows[b * p.snaps + s];
      if (sr > r0 && sr < r1) r1 = sr;
    }
    const int m = r1 - r0;
    // ---- rows -> shared memory (zeros outside)
    constexpr int CQ = DK / 8;
    for (int i = tid; i < kMlRows * CQ; i += 128) {
      const int r = i / CQ, c = (i % CQ) * 8;
      const bool live = r < m && c < D;
      const long long t = q0 + r0 + min(r, m - 1);
      const int cc = live ? c : 0;
      cp_async16(aq + (r * QS + c) * 2, p.q + t * p.ldq + head * D + cc, live);
      cp_async16(ak + (r * QS + c) * 2, p.k + t * p.ldk + head * D + cc, live);
    }
    for (int i = tid; i < kMlRows * 8; i += 128) {
      const int r = i >> 3, c = (i & 7) * 8;
      const bool live = r < m && c0 + c < V;
      const long long t = q0 + r0 + min(r, m - 1);
      cp_async16(av + (r * kMlVS + c) * 2, p.v + t * p.ldv + head * V + (live ? c0 + c : 0), live);
    }
    cp_async_commit();
    if (warp == 0) {                           // prefix sum of la over the chunk, two rows per lane
      const int ra = 2 * lane, rb = ra + 1;
      const long long ta = (long long)(q0 + r0) * p.H + head;
      const float xa = ra < m ? p.la[ta + (long long)ra * p.H] : 0.f, xb = rb < m ? p.la[ta + (long long)rb * p.H] : 0.f;
      float s = xa + xb;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += up;
      }
      const float total = __shfl_sync(0xffffffffu, s, 31);
      const float la_ = ra < m ? p.lb[ta + (long long)ra * p.H] : -INFINITY, lb_ = rb < m ? p.lb[ta + (long long)rb * p.H] : -INFINITY;
      sm.cum[ra] = s - xb; sm.cum[rb] = s;
      sm.lb[ra] = la_; sm.lb[rb] = lb_;
      sm.w[ra] = ra < m ? expf(total - (s - xb) + la_) : 0.f;
      sm.w[rb] = rb < m ? expf(total - s + lb_) : 0.f;
    }
    cp_async_wait<0>();
    __syncthreads();
    const float total = sm.cum[kMlRows - 1];   // rows past the end add nothing

    // ---- P = scale Q K^T weighted: this warp's 16 query rows against the keys up to them
    {
      float acc[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < DK / 16; ++kk) {
        uint32_t a[4];
        ldsm4(aq + ((warp * 16 + a_row) * QS + kk * 16 + a_col) * 2, a);
#pragma unroll
        for (int jj = 0; jj < 4; ++jj) {
          if (jj > warp) break;                // keys of later rows
          uint32_t bb[4];
          ldsm4(ak + ((jj * 16 + b_row) * QS + kk * 16 + b_col) * 2, bb);
          mma16816(acc[2 * jj], a, bb[0], bb[1]);
          mma16816(acc[2 * jj + 1], a, bb[2], bb[3]);
        }
      }
      const int ia = warp * 16 + g, ib = ia + 8;
      const float ca = sm.cum[ia], cb = sm.cum[ib];
      float sa = 0.f, sb = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int k0 = j * 8 + 2 * t4, k1 = k0 + 1;
        const float u0 = sm.lb[k0] - sm.cum[k0], u1 = sm.lb[k1] - sm.cum[k1];
        const float p00 = k0 <= ia ? acc[j][0] * p.scale * exp2f((ca + u0) * LOG2E) : 0.f;
        const float p01 = k1 <= ia ? acc[j][1] * p.scale * exp2f((ca + u1) * LOG2E) : 0.f;
        const float p10 = k0 <= ib ? acc[j][2] * p.scale * exp2f((cb + u0) * LOG2E) : 0.f;
        const float p11 = k1 <= ib ? acc[j][3] * p.scale * exp2f((cb + u1) * LOG2E) : 0.f;
        sa += p00 + p01;
        sb += p10 + p11;
        uint32_t hi, lo;
        split_bf16x2(p00, p01, hi, lo);
        *reinterpret_cast<uint32_t*>(&sm.ph[ia * kMlPS + k0]) = hi;
        *reinterpret_cast<uint32_t*>(&sm.pl[ia * kMlPS + k0]) = lo;
        split_bf16x2(p10, p11, hi, lo);
        *reinterpret_cast<uint32_t*>(&sm.ph[ib * kMlPS + k0]) = hi;
        *reinterpret_cast<uint32_t*>(&sm.pl[ib * kMlPS + k0]) = lo;
      }
      if (owner) {
        sa += __shfl_xor_sync(0xffffffffu, sa, 1); sa += __shfl_xor_sync(0xffffffffu, sa, 2);
        sb += __shfl_xor_sync(0xffffffffu, sb, 1); sb += __shfl_xor_sync(0xffffffffu, sb, 2);
        if (t4 == 0) { sm.rowsum[ia] = sa; sm.rowsum[ib] = sb; }
      }
    }
    // ---- num^T, the state's part: [16 channels x 64 rows] = S^T Q^T
    float o[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t ah[4], al[4];
      split_bf16x2(S[2 * kk][0], S[2 * kk][1], ah[0], al[0]);
      split_bf16x2(S[2 * kk][2], S[2 * kk][3], ah[1], al[1]);
      split_bf16x2(S[2 * kk + 1][0], S[2 * kk + 1][1], ah[2], al[2]);
      split_bf16x2(S[2 * kk + 1][2], S[2 * kk + 1][3], ah[3], al[3]);
#pragma unroll
      for (int jj = 0; jj < 4; ++jj) {
        uint32_t bb[4];
        ldsm4(aq + ((jj * 16 + b_row) * QS + kk * 16 + b_col) * 2, bb);
        mma16816(o[2 * jj], ah, bb[0], bb[1]);
        mma16816(o[2 * jj], al, bb[0], bb[1]);
        mma16816(o[2 * jj + 1], ah, bb[2], bb[3]);
        mma16816(o[2 * jj + 1], al, bb[2], bb[3]);
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float ga = p.scale * exp2f(sm.cum[j * 8 + 2 * t4] * LOG2E), gb = p.scale * exp2f(sm.cum[j * 8 + 2 * t4 + 1] * LOG2E);
      o[j][0] *= ga; o[j][1] *= gb; o[j][2] *= ga; o[j][3] *= gb;
    }
    __syncthreads();                           // P is complete
    // ---- num^T += V^T P^T
    uint32_t vf[4][4];                         // V^T fragments of this warp's 16 channels, kept for the state update
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      // A of [channel][token] out of rows [token][channel]: matrices (token half, channel half) -> a0, a1, a2, a3
      uint32_t x[4];
      ldsm4t(av + ((kk * 16 + a_row) * kMlVS + warp * 16 + a_col) * 2, x);
      vf[kk][0] = x[0]; vf[kk][1] = x[2]; vf[kk][2] = x[1]; vf[kk][3] = x[3];
#pragma unroll
      for (int jj = 0; jj < 4; ++jj) {
        if (jj < kk) continue;                 // query rows before these keys
        uint32_t bb[4];
        ldsm4(aph + ((jj * 16 + b_row) * kMlPS + kk * 16 + b_col) * 2, bb);
        mma16816(o[2 * jj], vf[kk], bb[0], bb[1]);
        mma16816(o[2 * jj + 1], vf[kk], bb[2], bb[3]);
        ldsm4(apl + ((jj * 16 + b_row) * kMlPS + kk * 16 + b_col) * 2, bb);
        mma16816(o[2 * jj], vf[kk], bb[0], bb[1]);
        mma16816(o[2 * jj + 1], vf[kk], bb[2], bb[3]);
      }
    }
    {
      __nv_bfloat16* so = sm.o[warp];
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) so[(j * 8 + 2 * t4 + (e & 1)) * 24 + g + 8 * (e >> 1)] = __float2bfloat16_rn(o[j][e]);
      __syncwarp();
      const int ch = c0 + warp * 16;
#pragma unroll
      for (int i = lane; i < kMlRows * 2; i += 32) {
        const int r = i >> 1, c = (i & 1) * 8;
        if (r < m && ch + c < V)
          *reinterpret_cast<uint4*>(p.out + (long long)(q0 + r0 + r) * p.ldo + head * V + ch + c) = *reinterpret_cast<const uint4*>(so + r * 24 + c);
      }
      __syncwarp();
    }
    // ---- denominators and the normaliser (one CTA per head)
    if (owner) {
      const int r = tid >> 1, half = tid & 1;  // two threads per row
      float dot = 0.f;
      const __nv_bfloat16* qr = sm.q + r * QS + half * (DK / 2);
#pragma unroll 4
      for (int c = 0; c < DK / 2; c += 8) {
        float f[8];
        load_vec<8>(qr + c, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) dot = fmaf(f[i], sm.n[half * (DK / 2) + c + i], dot);
      }
      dot += __shfl_xor_sync(0xffffffffu, dot, 1);
      if (half == 0 && r < m) {
        const long long t = (long long)(q0 + r0 + r) * p.H + head;
        const float d = sm.rowsum[r] + dot * p.scale * expf(sm.cum[r]);
        p.den[t] = fmaxf(fabsf(d), expf(-p.top[t])) + kMlstmEps;
      }
      __syncthreads();                         // uniform: `owner` is the whole CTA
      const float keep = expf(total);
      for (int c = tid; c < DK; c += 128) {
        float acc = sm.n[c] * keep;
        for (int j = 0; j < m; ++j) acc = fmaf(sm.w[j], __bfloat162float(sm.k[j * QS + c]), acc);
        sm.n[c] = acc;
      }
    }
    // ---- S^T = e^total S^T + (w V)^T K
    {
      const float keep = expf(total);
#pragma unroll
      for (int j = 0; j < KT; ++j) { S[j][0] *= keep; S[j][1] *= keep; S[j][2] *= keep; S[j][3] *= keep; }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t ah[4], al[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {          // tokens 2 t4, 2 t4 + 1 (+ 8 for the upper k half)
          const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&vf[kk][e]));
          const int tok = kk * 16 + 2 * t4 + 8 * (e >> 1);
          split_bf16x2(f.x * sm.w[tok], f.y * sm.w[tok + 1], ah[e], al[e]);
        }
#pragma unroll
        for (int j = 0; j < KT / 2; ++j) {
          uint32_t x[4];
          ldsm4t(ak + ((kk * 16 + a_row) * QS + j * 16 + a_col) * 2, x);
          mma16816(S[2 * j], ah, x[0], x[1]);
          mma16816(S[2 * j], al, x[0], x[1]);
          mma16816(S[2 * j + 1], ah, x[2], x[3]);
          mma16816(S[2 * j + 1], al, x[2], x[3]);
        }
      }
    }
    __syncthreads();                           // the chunk's rows are free, n is complete
    for (int s = 0; s < p.snaps; ++s)
      if (p.snap_rows[b * p.snaps + s] == r1) save(p.snap_slots[b * p.snaps + s]);
    r0 = r1;
  }
  if (p.commit) save(slot);
}

template <int DK>
static int launch_mlstm_chunk(const MlstmChunkParams& p, int B, cudaStream_t st) {
  constexpr int smem = (int)sizeof(MlstmSmem<DK>);
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(mlstm_chunk_kernel<DK>), smem) != cudaSuccess) return -20;
  mlstm_chunk_kernel<DK><<<dim3(p.H, (p.V + kMlCols - 1) / kMlCols, B), 128, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

template <typename T>
static int mlstm(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const float* la, const float* lb,
                 const float* top, float q_scale, float* h, void* out, long long ldo, float* den, const int* qsl, const int* slots,
                 const unsigned char* has, const int* limit, const int* snap_rows, const int* snap_slots, int snaps, int B, int H, int V,
                 int D, int commit, int one_row, cudaStream_t st) {
  ScanParams<T> p = {};
  p.a = reinterpret_cast<const T*>(q); p.lda = ldq; p.b = reinterpret_cast<const T*>(k); p.ldb = ldk;
  p.c = reinterpret_cast<const T*>(v); p.ldc = ldv; p.la = la; p.lb = lb; p.top = top; p.den = den; p.q_scale = q_scale;
  fill_batch(p, h, out, ldo, qsl, slots, has, limit, snap_rows, snap_slots, snaps, H, V + 1, D, 1, commit);
  return scan<T, kMlstm>(p, B, one_row, st);
}

}  // namespace atlas

using namespace atlas;
using bf16 = __nv_bfloat16;

// raw [T, 2 H] fp32; la, lb, top [T, H]; m [slots, H] is read (live slots) and, with `commit`, advanced
extern "C" int atlas_mlstm_gates(const float* raw, long long ld, const float* bias, float cap, float* m, float* la, float* lb, float* top,
                                 const int* qsl, const int* slots, const unsigned char* has, const int* limit, const int* snap_rows,
                                 const int* snap_slots, int snaps, int B, int H, int commit, void* stream) {
  if (B <= 0) return 0;
  if (H < 1 || !(cap > 0.f)) return -1;
  MlstmGateParams p = {raw, ld, bias, cap, m, la, lb, top, qsl, slots, has, limit, snap_rows, snap_slots, snaps, H, commit};
  launch_chain_if(true, mlstm_gates_kernel, dim3((H + 3) / 4, B), dim3(128), 0, reinterpret_cast<cudaStream_t>(stream), p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

// mLSTM memory (sequential form): la, lb, top [T, H] from atlas_mlstm_gates; q may be null (state only); h [slots, H, V + 1, D]
extern "C" int atlas_mlstm_scan(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const float* la,
                                const float* lb, const float* top, float q_scale, float* h, void* out, long long ldo, float* den,
                                const int* qsl, const int* slots, const unsigned char* has, const int* limit, const int* snap_rows,
                                const int* snap_slots, int snaps, int B, int H, int V, int D, int commit, int one_row, int f32,
                                void* stream) {
  if (out && !den) return -4;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? mlstm<float>(q, ldq, k, ldk, v, ldv, la, lb, top, q_scale, h, out, ldo, den, qsl, slots, has, limit, snap_rows, snap_slots,
                            snaps, B, H, V, D, commit, one_row, st)
             : mlstm<bf16>(q, ldq, k, ldk, v, ldv, la, lb, top, q_scale, h, out, ldo, den, qsl, slots, has, limit, snap_rows, snap_slots,
                           snaps, B, H, V, D, commit, one_row, st);
}

// The chunked form (bf16).  Returns 1 for shapes and alignments it does not take (nothing launched): the caller uses the scan.
extern "C" int atlas_mlstm_chunk(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const float* la,
                                 const float* lb, const float* top, float scale, float* h, void* out, long long ldo, float* den,
                                 const int* qsl, const int* slots, const unsigned char* has, const int* snap_rows, const int* snap_slots,
                                 int snaps, int B, int H, int V, int D, int commit, void* stream) {
  if (B <= 0) return 0;
  if (D > 256 || D % 8 || V % 8 || ldq % 8 || ldk % 8 || ldv % 8 || ldo % 8) return 1;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(out)) & 15) return 1;
  MlstmChunkParams p = {reinterpret_cast<const bf16*>(q), ldq, reinterpret_cast<const bf16*>(k), ldk, reinterpret_cast<const bf16*>(v), ldv,
                        la, lb, top, scale, h, reinterpret_cast<bf16*>(out), ldo, den, qsl, slots, has, snap_rows, snap_slots, snaps, H, V, D,
                        commit};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (D <= 64) return launch_mlstm_chunk<64>(p, B, st);
  if (D <= 128) return launch_mlstm_chunk<128>(p, B, st);
  return launch_mlstm_chunk<256>(p, B, st);
}
