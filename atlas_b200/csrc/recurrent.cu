// Mamba-2 and WKV recurrences (kernels in linear_scan.cuh).  Activations are bf16 or fp32 (template parameter T).
// Reference ops replaced: kernels/gb10/common/mamba2_ssm_decode.cu, mamba2_ssd_chunk.cu.
#include "common.cuh"
#include "host_api.h"
#include "linear_scan.cuh"
#include "vec_io.cuh"

namespace atlas {

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
