// One decode step of the recurrences in state_scan.cu (same state, same equations), one CTA per (row, head).
//
// The step is bound by the state's bytes: dim x vdim fp32 read and written per row and head.  A thread holds four neighbouring
// columns of RPT rows; all loads are asked for before anything is computed, and the other inputs are prepared while the state
// travels:
// for the gated delta rule the short convolution with SiLU of this head's q, k and v channels (csrc/gated_glue.cu has it as a
// kernel of its own), unit norms, step size and decay.  Then one pass gives a = k S and b = q S, partial sums meet in shared
// memory, e = beta (v - g a), o = g b + (k . q) e, and g S + k (x) e is written to the other half of the slot.  The gated
// delta rule's output is normed per head, gated and scaled here as well; lightning's, whose norm spans the heads, goes out
// as fp32.

#include "glue.cuh"

namespace b200 {

constexpr int kStepThreads = 256;

struct StepParams {
  const void* act;     // DELTA: inputs of the convolution; else activated rows.  [rows, ld]
  int ld, q_off, k_off, v_off;
  const void* conv_w;  // DELTA: [taps, ld]
  void* ring;          // DELTA: [num_slots, taps, ld]
  int taps;
  const float* ba;
  const float* a_log;
  const float* dt_bias;
  const float* decay;
  float* state;
  const int* slots;
  const int* positions;
  float* o;               // !DELTA: [rows, heads, vdim]
  const void* gate;       // DELTA: [rows, heads, vdim]
  const float* norm;      // DELTA: [vdim]
  void* out;              // DELTA: rows out_ld apart, head h at column h * vdim
  int out_ld, norm_size;
  float eps, out_scale, q_scale;
  int* err;
  int rows, heads, qk_heads, dim, vdim, num_slots;
};

__device__ __forceinline__ float step_log_decay(float a_log, float a, float dt_bias) {
  const float z = a + dt_bias;
  return -expf(a_log) * (z > 20.f ? z : log1pf(expf(z)));
}

// Sum over the CTA; every thread gets it.  `red` has a float per warp.
__device__ __forceinline__ float cta_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < kStepThreads / 32; ++i) s += red[i];
  return s;
}

template <typename T, int RPT, bool DELTA>
__global__ void __launch_bounds__(kStepThreads)
state_step_kernel(const StepParams p) {
  extern __shared__ float st_sm[];  // k[dim], q[dim], v[vdim], part[2][row groups][vdim], u[vdim]
  __shared__ float red[kStepThreads / 32], sums[kStepThreads / 32][3];
  grid_dep_wait();
  grid_dep_launch();
  const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x;
  const int pos = p.positions[row], slot = p.slots[row];
  if (slot < 0 || slot >= p.num_slots || pos < 0) {
    if (tid == 0) set_error(p.err, kErrDevBadBlockId);
    return;
  }
  const int cgs = p.vdim / 4, rgs = kStepThreads / cgs;  // column groups of four, row groups
  const int rg = tid / cgs, c = (tid - rg * cgs) * 4;
  const bool in = rg < rgs;
  const size_t half = static_cast<size_t>(p.heads) * p.dim * p.vdim;
  float* st = p.state + static_cast<size_t>(slot) * 2 * half + static_cast<size_t>(h) * p.dim * p.vdim + c;
  const float* src = st + ((pos - 1) & 1) * half;
  float* ks = st_sm;
  float* qs = ks + p.dim;
  float* vs = qs + p.dim;
  float* part = vs + p.vdim;
  float* us = part + 2 * rgs * p.vdim;
  const int per = p.heads / p.qk_heads, qh = h / per;
  const T* act = static_cast<const T*>(p.act) + static_cast<size_t>(row) * p.ld;
  // q, k, v of this head, one value per thread and turn
  const int n = 2 * p.dim + p.vdim;
  float kk = 0.f, qq = 0.f, b_in = 0.f, a_in = 0.f, alog = 0.f, dtb = 0.f;
  if (DELTA) {
    const float* ba = p.ba + static_cast<size_t>(row) * 2 * p.heads;
    b_in = ba[h];
    a_in = ba[p.heads + h];
    alog = p.a_log[h];
    dtb = p.dt_bias[h];
  }
  const T* conv_w = static_cast<const T*>(p.conv_w);
  T* ring = DELTA && p.taps > 1 ? static_cast<T*>(p.ring) + static_cast<size_t>(slot) * p.taps * p.ld : nullptr;
  const auto channel = [&](int i) {
    return i < p.dim ? p.q_off + qh * p.dim + i : i < 2 * p.dim ? p.k_off + qh * p.dim + i - p.dim : p.v_off + h * p.vdim + i - 2 * p.dim;
  };
  // taps whose loads are in flight together, for two channels of the thread
  constexpr int kNear = 4;
  T x_in[2], w_in[2][kNear], h_in[2][kNear];
  const int pos_row = DELTA && p.taps > 1 ? pos % p.taps : 0;
  const auto ask = [&](int i0) {
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = i0 + u * kStepThreads;
      if (i >= n) break;
      const int ch = channel(i);
      x_in[u] = act[ch];
      if (DELTA) {
#pragma unroll
        for (int j = 0; j < kNear; ++j) {  // j positions back
          const int r = pos_row - j;       // row of the ring
          w_in[u][j] = j < p.taps ? conv_w[static_cast<size_t>(p.taps - 1 - j) * p.ld + ch] : from_f32<T>(0.f);
          h_in[u][j] = j > 0 && j < p.taps && pos >= j ? ring[static_cast<size_t>(r < 0 ? r + p.taps : r) * p.ld + ch] : from_f32<T>(0.f);
        }
      }
    }
  };
  ask(tid);  // ahead of the state, which is many times as long
  // the head norm's weight and the gate of this thread's output column
  float norm_w = 0.f, gate_v = 0.f;
  if (DELTA && tid < p.vdim) {
    norm_w = p.norm[tid];
    gate_v = to_f32<T>(static_cast<const T*>(p.gate)[(static_cast<size_t>(row) * p.heads + h) * p.vdim + tid]);
  }
  float4 S[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = rg + i * rgs;
    S[i] = in && pos > 0 && r < p.dim ? __ldcs(reinterpret_cast<const float4*>(src + static_cast<size_t>(r) * p.vdim))
                                      : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int i0 = tid; i0 < n; i0 += 2 * kStepThreads) {
    if (i0 != tid) ask(i0);
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = i0 + u * kStepThreads;
      if (i >= n) break;
      float x = to_f32<T>(x_in[u]);
      if (DELTA) {
        const int ch = channel(i);
        float acc = 0.f;
        for (int j = 0; j + kNear < p.taps; ++j) {
          const int at = pos - p.taps + 1 + j;
          if (at >= 0)
            acc = fmaf(to_f32<T>(conv_w[static_cast<size_t>(j) * p.ld + ch]), to_f32<T>(ring[static_cast<size_t>(at % p.taps) * p.ld + ch]), acc);
        }
#pragma unroll
        for (int j = kNear - 1; j > 0; --j) acc = fmaf(to_f32<T>(w_in[u][j]), to_f32<T>(h_in[u][j]), acc);
        acc = fmaf(to_f32<T>(w_in[u][0]), x, acc);
        // the heads that share q and k write the same value once: the first of them
        if (ring != nullptr && (i >= 2 * p.dim || h == qh * per)) ring[static_cast<size_t>(pos_row) * p.ld + ch] = x_in[u];
        x = to_f32<T>(from_f32<T>(silu_as<T>(acc)));
      }
      if (i < p.dim) {
        qs[i] = x;
        qq = fmaf(x, x, qq);
      } else if (i < 2 * p.dim) {
        ks[i - p.dim] = x;
        kk = fmaf(x, x, kk);
      } else {
        vs[i - 2 * p.dim] = x;
      }
    }
  }
  if (DELTA) {
    kk = warp_sum(kk);
    qq = warp_sum(qq);
    if ((tid & 31) == 0) {
      sums[tid >> 5][0] = kk;
      sums[tid >> 5][1] = qq;
    }
  }
  __syncthreads();
  float dot = 0.f;
  for (int i = tid; i < p.dim; i += kStepThreads) dot = fmaf(ks[i], qs[i], dot);
  dot = warp_sum(dot);
  if ((tid & 31) == 0) sums[tid >> 5][2] = dot;
  float ik = 1.f, iq = 1.f, g, beta = 1.f;
  if (DELTA) {
    kk = qq = 0.f;
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; ++i) {
      kk += sums[i][0];
      qq += sums[i][1];
    }
    ik = 1.f / sqrtf(kk + 1e-6f);
    iq = p.q_scale / sqrtf(qq + 1e-6f);
    beta = sigmoid_of(b_in);
    g = expf(step_log_decay(alog, a_in, dtb));
  } else {
    g = p.decay[h];
  }
  if (in) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = rg + i * rgs;
      if (r >= p.dim) break;
      const float kv = ks[r], qv = qs[r];
      if (DELTA) {
        a.x = fmaf(kv, S[i].x, a.x);
        a.y = fmaf(kv, S[i].y, a.y);
        a.z = fmaf(kv, S[i].z, a.z);
        a.w = fmaf(kv, S[i].w, a.w);
      }
      b.x = fmaf(qv, S[i].x, b.x);
      b.y = fmaf(qv, S[i].y, b.y);
      b.z = fmaf(qv, S[i].z, b.z);
      b.w = fmaf(qv, S[i].w, b.w);
    }
    if (DELTA) *reinterpret_cast<float4*>(part + rg * p.vdim + c) = a;
    *reinterpret_cast<float4*>(part + (rgs + rg) * p.vdim + c) = b;
  }
  __syncthreads();
  dot = 0.f;
#pragma unroll
  for (int i = 0; i < kStepThreads / 32; ++i) dot += sums[i][2];
  dot *= ik * iq;
  float ss = 0.f;
  for (int j = tid; j < p.vdim; j += kStepThreads) {
    float a = 0.f, b = 0.f;
    for (int r = 0; r < rgs; ++r) {
      if (DELTA) a += part[r * p.vdim + j];
      b += part[(rgs + r) * p.vdim + j];
    }
    const float u = DELTA ? beta * (vs[j] - g * ik * a) : vs[j];
    const float o = fmaf(dot, u, g * iq * b);
    us[j] = u * ik;  // the update's k is the raw one
    if (DELTA) {
      vs[j] = o;
      ss = fmaf(o, o, ss);
    } else {
      p.o[(static_cast<size_t>(row) * p.heads + h) * p.vdim + j] = o;
    }
  }
  __syncthreads();
  if (in) {
    float* dst = st + (pos & 1) * half;
    const float4 u = *reinterpret_cast<const float4*>(us + c);
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = rg + i * rgs;
      if (r >= p.dim) break;
      const float kv = ks[r];
      float4 v;
      v.x = fmaf(kv, u.x, g * S[i].x);
      v.y = fmaf(kv, u.y, g * S[i].y);
      v.z = fmaf(kv, u.z, g * S[i].z);
      v.w = fmaf(kv, u.w, g * S[i].w);
      __stcs(reinterpret_cast<float4*>(dst + static_cast<size_t>(r) * p.vdim), v);
    }
  }
  if (DELTA) {
    const float inv = p.out_scale / sqrtf(cta_sum(ss, red) / static_cast<float>(p.norm_size) + p.eps);
    T* out = static_cast<T*>(p.out) + static_cast<size_t>(row) * p.out_ld + static_cast<size_t>(h) * p.vdim;
    for (int j = tid; j < p.vdim; j += kStepThreads) {
      if (j >= kStepThreads) {
        norm_w = p.norm[j];
        gate_v = to_f32<T>(static_cast<const T*>(p.gate)[(static_cast<size_t>(row) * p.heads + h) * p.vdim + j]);
      }
      out[j] = from_f32<T>(vs[j] * inv * norm_w * gate_v);
    }
  }
}

static int step_rows_per_thread(int dim, int vdim) {
  const int rgs = vdim % 4 == 0 && vdim <= 4 * kStepThreads ? kStepThreads / (vdim / 4) : 0;
  return rgs > 0 ? (dim + rgs - 1) / rgs : 1 << 30;
}

template <typename T, bool DELTA>
static int launch_step(const StepParams& p, cudaStream_t st) {
  const int rpt = step_rows_per_thread(p.dim, p.vdim), rgs = kStepThreads / (p.vdim / 4);
  const size_t smem = (2 * static_cast<size_t>(p.dim) + 2 * p.vdim + 2 * static_cast<size_t>(rgs) * p.vdim) * 4;
#define B200_STEP(RPT)                                                                                                   \
  B200_CUDA(launch_overlapped(state_step_kernel<T, RPT, DELTA>, dim3(p.heads, p.rows), dim3(kStepThreads), smem, st, p))
  if (rpt <= 4) B200_STEP(4);
  else if (rpt <= 8) B200_STEP(8);
  else if (rpt <= 16) B200_STEP(16);
  else B200_STEP(32);
#undef B200_STEP
  return 0;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_state_step_supported(int dim, int vdim) {
  // the head's vectors and partial sums stay below the 48 KiB of shared memory a kernel has without asking for more
  return dim > 0 && vdim > 0 && dim % 4 == 0 && vdim % 4 == 0 && vdim <= 1024 && step_rows_per_thread(dim, vdim) <= 32 &&
         (2 * dim + 2 * vdim + 2 * 4 * kStepThreads) * 4 <= 46 * 1024;
}

extern "C" int b200_state_step(const void* act, int ld, int q_off, int k_off, int v_off, const void* conv_w, void* ring, int taps,
                               const float* ba, const float* a_log, const float* dt_bias, const float* decay, float* state,
                               const int32_t* slots, const int32_t* positions, float* o, const void* gate, const float* norm,
                               void* out, int out_ld, int norm_size, float eps, float out_scale, void* status_word, int num_rows,
                               int heads, int qk_heads, int dim, int vdim, int num_slots, float q_scale, int dtype, void* stream) {
  B200_REQUIRE(act && state && slots && positions, "state_step: null pointer");
  B200_REQUIRE((decay && o) || (ba && a_log && dt_bias && conv_w && taps >= 1 && (taps == 1 || ring) && gate && norm && out && norm_size > 0),
               "state_step: a fixed decay and fp32 rows, or all that the gated delta rule needs");
  B200_REQUIRE(num_rows >= 0 && num_rows <= 65535 && heads > 0 && qk_heads > 0 && heads % qk_heads == 0 && num_slots > 0 &&
                   b200_state_step_supported(dim, vdim),
               "state_step: %d rows, %d heads over %d, state %d x %d", num_rows, heads, qk_heads, dim, vdim);
  B200_REQUIRE(q_off >= 0 && k_off >= 0 && v_off >= 0 && q_off + qk_heads * dim <= ld && k_off + qk_heads * dim <= ld &&
                   v_off + heads * vdim <= ld && (decay || out_ld >= heads * vdim),
               "state_step: q, k and v do not fit rows of %d", ld);
  B200_REQUIRE((reinterpret_cast<uintptr_t>(state) & 15) == 0, "state_step: the state must be 16-byte aligned");
  B200_GLUE_DTYPE("state_step");
  if (num_rows == 0) return 0;
  const StepParams p{act, ld, q_off, k_off, v_off, conv_w, ring, taps, ba, a_log, dt_bias, decay, state, slots, positions, o, gate,
                     norm, out, out_ld, norm_size, eps, out_scale, q_scale, static_cast<int*>(status_word), num_rows, heads,
                     qk_heads, dim, vdim, num_slots};
  if (dtype == 0)
    return decay ? launch_step<__nv_bfloat16, false>(p, as_stream(stream)) : launch_step<__nv_bfloat16, true>(p, as_stream(stream));
  return decay ? launch_step<float, false>(p, as_stream(stream)) : launch_step<float, true>(p, as_stream(stream));
}
