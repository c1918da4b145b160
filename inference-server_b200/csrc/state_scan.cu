// Recurrences over a matrix state per head (csrc of the layer-list decoders' lightning attention and gated delta rule):
//
//     S_t = g_t S_{t-1} + k_t (x) e_t,    e_t = DELTA ? beta_t (v_t - g_t k_t S_{t-1}) : v_t,    o_t = q_t S_t
//
// with row vectors, (x) the outer product and S [dim, vdim] fp32, kept from step to step in a slot per sequence:  state [slots, 2, heads, dim, vdim].  The state
// after position p is in half p & 1 of the slot, so a decode step reads one half and writes the other and may be run
// again; position 0 starts from zeros whatever the slot holds, so a slot needs no clearing when it changes hands.
//
// DELTA: q and k are made unit vectors, q times q_scale; beta = sigmoid(ba[:, h]), g = exp(-exp(a_log) softplus(ba[:, H + h]
// + dt_bias)).  Otherwise g = decay[h] and q, k are taken as they are.
//
// The columns of S do not meet, so a head's columns are spread over warps.  Scan kernel: a warp owns 4 * CPL columns; its
// lanes are 8 row groups x 4 column groups, a lane holds 4 * R4 rows of CPL columns in registers.  With a = k S, b = q S of the
// state before the token, e = beta (v - g a) and o = g b + (k . q) e: both products are taken in one pass over the state
// and reduced together, and the update follows.

#include "glue.cuh"

namespace b200 {

struct ScanParams {
  const void* act;    // [rows, ld]: q heads, k heads, v heads
  int ld, q_off, k_off, v_off;
  const float* ba;    // DELTA: [rows, 2 * heads]
  const float* a_log;
  const float* dt_bias;
  const float* decay; // !DELTA: [heads]
  float* state;
  const int* slots;
  const int* positions;
  float* o;           // [rows, heads, vdim]
  int* err;
  int rows, chunk;    // chunk: all rows are one sequence, positions[0] on; else a sequence per row
  int heads, qk_heads, dim, vdim, num_slots;
  float q_scale;
};

constexpr int kScanTokens = 16;  // tokens staged at a time

__device__ __forceinline__ float delta_log_decay(float a_log, float a, float dt_bias) {
  const float z = a + dt_bias;
  const float sp = z > 20.f ? z : log1pf(expf(z));
  return -expf(a_log) * sp;
}

template <typename T, int R4, int CPL, bool DELTA>
__global__ void __launch_bounds__(128)
state_scan_kernel(const ScanParams p) {
  constexpr int kDim = 32 * R4;          // rows held, >= dim
  constexpr int kCols = 16 * CPL;        // columns per CTA
  __shared__ __align__(16) float ks[kScanTokens][kDim], qs[kScanTokens][kDim];
  __shared__ float vs[kScanTokens][kCols], gs[kScanTokens], bs[kScanTokens], kq[kScanTokens];
  grid_dep_wait();
  grid_dep_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rg = lane >> 2, cg = lane & 3;
  const int h = blockIdx.y, seq = blockIdx.z;
  const int col_local = warp * 4 * CPL + cg * CPL, col = blockIdx.x * kCols + col_local;
  const int qh = h / (p.heads / p.qk_heads);
  const int row0 = p.chunk ? 0 : seq, n = p.chunk ? p.rows : 1;
  const int first = p.positions[row0], slot = p.slots[row0];
  if (slot < 0 || slot >= p.num_slots || first < 0) {
    if (threadIdx.x == 0) set_error(p.err, kErrDevBadBlockId);
    return;
  }
  const size_t half = static_cast<size_t>(p.heads) * p.dim * p.vdim;
  float* st = p.state + static_cast<size_t>(slot) * 2 * half + static_cast<size_t>(h) * p.dim * p.vdim;
  const T* act = static_cast<const T*>(p.act);

  float S[4 * R4][CPL];
  {
    const float* src = st + ((first - 1) & 1) * half;
#pragma unroll
    for (int i = 0; i < 4 * R4; ++i) {
      const int r = (i >> 2) * 32 + rg * 4 + (i & 3);
#pragma unroll
      for (int c = 0; c < CPL; ++c)
        S[i][c] = first > 0 && r < p.dim && col + c < p.vdim ? src[static_cast<size_t>(r) * p.vdim + col + c] : 0.f;
    }
  }
  for (int t0 = 0; t0 < n; t0 += kScanTokens) {
    const int cnt = min(kScanTokens, n - t0);
    __syncthreads();  // the tokens before have been read
    for (int t = warp; t < cnt; t += 4) {
      const size_t row = static_cast<size_t>(row0 + t0 + t);
      const T* kr = act + row * p.ld + p.k_off + qh * p.dim;
      const T* qr = act + row * p.ld + p.q_off + qh * p.dim;
      float kk = 0.f, qq = 0.f, dot = 0.f;
#pragma unroll
      for (int i = 0; i < R4; ++i) {
        const int r = i * 32 + lane;
        const float kv = r < p.dim ? to_f32<T>(kr[r]) : 0.f, qv = r < p.dim ? to_f32<T>(qr[r]) : 0.f;
        ks[t][r] = kv;
        qs[t][r] = qv;
        kk = fmaf(kv, kv, kk);
        qq = fmaf(qv, qv, qq);
        dot = fmaf(kv, qv, dot);
      }
      dot = warp_sum(dot);
      if (DELTA) {
        const float ik = 1.f / sqrtf(warp_sum(kk) + 1e-6f), iq = p.q_scale / sqrtf(warp_sum(qq) + 1e-6f);
#pragma unroll
        for (int i = 0; i < R4; ++i) {
          ks[t][i * 32 + lane] *= ik;
          qs[t][i * 32 + lane] *= iq;
        }
        dot *= ik * iq;
      }
      if (lane == 0) {
        kq[t] = dot;
        if (DELTA) {
          bs[t] = 1.f / (1.f + expf(-p.ba[row * 2 * p.heads + h]));
          gs[t] = expf(delta_log_decay(p.a_log[h], p.ba[row * 2 * p.heads + p.heads + h], p.dt_bias[h]));
        } else {
          gs[t] = p.decay[h];
        }
      }
    }
    for (int i = threadIdx.x; i < cnt * kCols; i += 128) {
      const int t = i / kCols, c = i - t * kCols, cc = blockIdx.x * kCols + c;
      vs[t][c] = cc < p.vdim ? to_f32<T>(act[static_cast<size_t>(row0 + t0 + t) * p.ld + p.v_off + h * p.vdim + cc]) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < cnt; ++t) {
      float a[CPL], b[CPL], kf[4 * R4];
#pragma unroll
      for (int c = 0; c < CPL; ++c) a[c] = b[c] = 0.f;
#pragma unroll
      for (int i = 0; i < R4; ++i) {
        const float4 k4 = *reinterpret_cast<const float4*>(&ks[t][i * 32 + rg * 4]);
        const float4 q4 = *reinterpret_cast<const float4*>(&qs[t][i * 32 + rg * 4]);
        kf[4 * i] = k4.x; kf[4 * i + 1] = k4.y; kf[4 * i + 2] = k4.z; kf[4 * i + 3] = k4.w;
        const float qf[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int c = 0; c < CPL; ++c) {
            if (DELTA) a[c] = fmaf(kf[4 * i + e], S[4 * i + e][c], a[c]);
            b[c] = fmaf(qf[e], S[4 * i + e][c], b[c]);
          }
      }
#pragma unroll
      for (int s = 4; s < 32; s <<= 1)
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          if (DELTA) a[c] += __shfl_xor_sync(0xffffffffu, a[c], s);
          b[c] += __shfl_xor_sync(0xffffffffu, b[c], s);
        }
      const float g = gs[t], dot = kq[t];
      float u[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        const float v = vs[t][col_local + c];
        u[c] = DELTA ? bs[t] * (v - g * a[c]) : v;
        b[c] = fmaf(dot, u[c], g * b[c]);
      }
#pragma unroll
      for (int i = 0; i < 4 * R4; ++i)
#pragma unroll
        for (int c = 0; c < CPL; ++c) S[i][c] = fmaf(kf[i], u[c], g * S[i][c]);
      if (rg == 0)
#pragma unroll
        for (int c = 0; c < CPL; ++c)
          if (col + c < p.vdim) p.o[(static_cast<size_t>(row0 + t0 + t) * p.heads + h) * p.vdim + col + c] = b[c];
    }
  }
  float* dst = st + ((first + n - 1) & 1) * half;
#pragma unroll
  for (int i = 0; i < 4 * R4; ++i) {
    const int r = (i >> 2) * 32 + rg * 4 + (i & 3);
#pragma unroll
    for (int c = 0; c < CPL; ++c)
      if (r < p.dim && col + c < p.vdim) dst[static_cast<size_t>(r) * p.vdim + col + c] = S[i][c];
  }
}

template <typename T, bool DELTA>
static int launch_scan(const ScanParams& p, cudaStream_t st) {
#define B200_SCAN(R4, CPL)                                                                                            \
  B200_CUDA(launch_overlapped(state_scan_kernel<T, R4, CPL, DELTA>,                                                   \
                              dim3((p.vdim + 16 * CPL - 1) / (16 * CPL), p.heads, p.chunk ? 1 : p.rows), dim3(128), 0, st, p))
  if (p.dim <= 32) B200_SCAN(1, 2);
  else if (p.dim <= 64) B200_SCAN(2, 2);
  else if (p.dim <= 128) B200_SCAN(4, 2);
  else if (p.dim <= 256) B200_SCAN(8, 2);
  else B200_SCAN(10, 1);
#undef B200_SCAN
  return 0;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_state_scan(const void* act, int ld, int q_off, int k_off, int v_off, const float* ba, const float* a_log,
                               const float* dt_bias, const float* decay, float* state, const int32_t* slots,
                               const int32_t* positions, float* o, void* status_word, int num_rows, int chunk, int heads,
                               int qk_heads, int dim, int vdim, int num_slots, float q_scale, int dtype, void* stream) {
  B200_REQUIRE(act && state && slots && positions && o, "state_scan: null pointer");
  B200_REQUIRE((decay != nullptr) != (ba && a_log && dt_bias), "state_scan: a fixed decay, or beta, a_log and dt_bias");
  B200_REQUIRE(num_rows >= 0 && heads > 0 && heads <= 65535 && qk_heads > 0 && heads % qk_heads == 0 && dim > 0 && dim <= 320 &&
                   vdim > 0 && num_slots > 0 && (chunk || num_rows <= 65535),
               "state_scan: %d rows, %d heads over %d, state %d x %d (at most 320 rows)", num_rows, heads, qk_heads, dim, vdim);
  B200_REQUIRE(q_off >= 0 && k_off >= 0 && v_off >= 0 && q_off + qk_heads * dim <= ld && k_off + qk_heads * dim <= ld &&
                   v_off + heads * vdim <= ld,
               "state_scan: q, k and v do not fit rows of %d", ld);
  B200_GLUE_DTYPE("state_scan");
  if (num_rows == 0) return 0;
  const ScanParams p{act, ld, q_off, k_off, v_off, ba, a_log, dt_bias, decay, state, slots, positions, o,
                     static_cast<int*>(status_word), num_rows, chunk, heads, qk_heads, dim, vdim, num_slots, q_scale};
  if (dtype == 0)
    return decay ? launch_scan<__nv_bfloat16, false>(p, as_stream(stream)) : launch_scan<__nv_bfloat16, true>(p, as_stream(stream));
  return decay ? launch_scan<float, false>(p, as_stream(stream)) : launch_scan<float, true>(p, as_stream(stream));
}
