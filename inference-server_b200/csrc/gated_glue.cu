// Small kernels of the gated layer-list decoders (Sefalorn; engine: layered.py) between the matrix products: residual add
// with an element-wise gate and layer norm (or RMS norm), mixing of query heads ahead of attention, the short convolution
// with SiLU in front of a recurrence, and the grouped norm and gate behind one.  Statistics, convolution sums and the
// residual are fp32; T is the type of the activations between kernels (bf16 or fp32).

#include "glue.cuh"

namespace b200 {

template <typename T>
__device__ __forceinline__ void store4(T* dst, const float4& v) {
  if constexpr (sizeof(T) == 2) {
    uint2 two;
    two.x = pack_bf16x2(v.x, v.y);
    two.y = pack_bf16x2(v.z, v.w);
    *reinterpret_cast<uint2*>(dst) = two;
  } else {
    *reinterpret_cast<float4*>(dst) = v;
  }
}

// What a sublayer left for the residual stream: rows of its own, or the experts' rows that the token's pairs point to.
template <typename T>
struct Pending {
  const T* dense;          // [M, ld]
  const T* expert_rows;    // [pairs, ld], with the three below
  const int* row_of_pair;  // [M, top_k], -1 = none
  const float* pair_weight;
  int top_k;
  const float* bias;       // [ld], added to the sublayer's result
  const T* gate;           // [M, ld], multiplies it
};

// x += (sublayer + bias) * gate; out = (x - mean) / sqrt(var + eps) * w (CENTER), or x / rms * w.  One CTA per row, eight
// columns per thread.
template <typename T, bool CENTER, int MAXT>
__global__ void __launch_bounds__(MAXT)
residual_norm_kernel(float* __restrict__ x, const Pending<T> p, const float* __restrict__ weight, float eps, int width,
                     int ld, T* __restrict__ out) {
  __shared__ float red[2][32];
  grid_dep_wait();
  grid_dep_launch();
  const int m = blockIdx.x, col = threadIdx.x * 8, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool in = col < ld;
  const size_t at = static_cast<size_t>(m) * ld + col;
  float f[8], w[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) f[j] = w[j] = 0.f;
  if (in) {
    load8<float>(x + at, f);
    load8<float>(weight + col, w);
    const bool any = p.dense != nullptr || p.expert_rows != nullptr;
    if (any) {
      Raw8<T> g;
      if (p.gate != nullptr) g.load(p.gate + at);
      float d[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) d[j] = 0.f;
      if (p.dense != nullptr) {
        load8<T>(p.dense + at, d);
      } else {
        for (int k0 = 0; k0 < p.top_k; k0 += 8) {  // eight pairs at a time: their rows are in flight together
          int rows[8];
          float pw[8];
          Raw8<T> raw[8];
#pragma unroll
          for (int u = 0; u < 8; ++u) {
            const bool have = k0 + u < p.top_k;
            rows[u] = have ? p.row_of_pair[static_cast<size_t>(m) * p.top_k + k0 + u] : -1;
            pw[u] = have ? p.pair_weight[static_cast<size_t>(m) * p.top_k + k0 + u] : 0.f;
          }
#pragma unroll
          for (int u = 0; u < 8; ++u)
            if (rows[u] >= 0) raw[u].load(p.expert_rows + static_cast<size_t>(rows[u]) * ld + col);
#pragma unroll
          for (int u = 0; u < 8; ++u) {
            if (rows[u] < 0) continue;
            float y[8];
            raw[u].get(y);
#pragma unroll
            for (int j = 0; j < 8; ++j) d[j] = fmaf(pw[u], y[j], d[j]);
          }
        }
      }
      if (p.bias != nullptr) {
        float b[8];
        load8<float>(p.bias + col, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) d[j] += b[j];
      }
      if (p.gate != nullptr) {
        float gf[8];
        g.get(gf);
#pragma unroll
        for (int j = 0; j < 8; ++j) d[j] *= gf[j];
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = col + j < width ? f[j] + d[j] : 0.f;
      store8<float>(x + at, f);
    }
  }
  const int warps = blockDim.x >> 5;
  float mean = 0.f;
  if (CENTER) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) s += f[j];
    s = warp_sum(s);
    if (lane == 0) red[0][warp] = s;
    __syncthreads();
    mean = warp_sum(lane < warps ? red[0][lane] : 0.f) / static_cast<float>(width);
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    f[j] = col + j < width ? f[j] - mean : 0.f;
    ss += f[j] * f[j];
  }
  ss = warp_sum(ss);
  if (lane == 0) red[1][warp] = ss;
  __syncthreads();
  const float inv = 1.f / sqrtf(warp_sum(lane < warps ? red[1][lane] : 0.f) / static_cast<float>(width) + eps);
  if (!in) return;
#pragma unroll
  for (int j = 0; j < 8; ++j) f[j] = f[j] * inv * w[j];
  store8<T>(out + at, f);
}

// out[m, h, c * D + d] = sum over the query heads g of kv head c of mix[h, g] * q[m, g, d]: with it, scores mixed over the
// heads are plain products with the keys of all kv heads side by side.  One CTA per (`rows_per` rows, kv head); a thread makes
// four columns of four heads.
template <typename T>
__global__ void __launch_bounds__(256)
mix_heads_kernel(const T* __restrict__ q, const float* __restrict__ mix, T* __restrict__ out, int num_rows, int rows_per,
                 int heads, int kv_heads, int D) {
  grid_dep_wait();
  grid_dep_launch();
  extern __shared__ float mh_sm[];
  const int c = blockIdx.y, per = heads / kv_heads;
  const int m0 = blockIdx.x * rows_per, rows = min(rows_per, num_rows - m0);
  const int hp = (heads + 3) & ~3, row_q = per * D;
  float* ms = mh_sm;             // [per, heads rounded up to 4]
  float* qs = mh_sm + per * hp;  // [rows, per, D]
  for (int i = threadIdx.x; i < per * hp; i += blockDim.x) {
    const int g = i / hp, h = i - g * hp;
    ms[i] = h < heads ? mix[static_cast<size_t>(h) * heads + c * per + g] : 0.f;
  }
  for (int x = threadIdx.x * 4; x < row_q; x += blockDim.x * 4) {
    const T* src = q + (static_cast<size_t>(m0) * heads + c * per) * D + x;
#pragma unroll 8
    for (int r = 0; r < rows; ++r) {
      const T* s = src + static_cast<size_t>(r) * heads * D;
      float4 v;
      if constexpr (sizeof(T) == 2) {
        const uint2 raw = *reinterpret_cast<const uint2*>(s);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        v = make_float4(a.x, a.y, b.x, b.y);
      } else {
        v = *reinterpret_cast<const float4*>(s);
      }
      *reinterpret_cast<float4*>(qs + r * row_q + x) = v;
    }
  }
  __syncthreads();
  const int d4 = D / 4, per_row = (hp / 4) * d4, items = rows * per_row;
  if (per <= 8) {  // a thread's mixing factors stay in registers over the rows
    for (int rest = threadIdx.x; rest < per_row; rest += blockDim.x) {
      const int h0 = rest / d4 * 4, d = (rest % d4) * 4;
      float4 a[8];
#pragma unroll
      for (int g = 0; g < 8; ++g)
        a[g] = g < per ? *reinterpret_cast<const float4*>(ms + g * hp + h0) : make_float4(0.f, 0.f, 0.f, 0.f);
      T* dst = out + ((static_cast<size_t>(m0) * heads + h0) * kv_heads + c) * D + d;
#pragma unroll 2
      for (int r = 0; r < rows; ++r) {
        float2 acc[4][2];
#pragma unroll
        for (int u = 0; u < 4; ++u) acc[u][0] = acc[u][1] = make_float2(0.f, 0.f);
#pragma unroll
        for (int g = 0; g < 8; ++g) {
          if (g >= per) break;
          const float4 v = *reinterpret_cast<const float4*>(qs + r * row_q + g * D + d);
          const float aa[4] = {a[g].x, a[g].y, a[g].z, a[g].w};
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            acc[u][0] = __ffma2_rn(make_float2(aa[u], aa[u]), make_float2(v.x, v.y), acc[u][0]);
            acc[u][1] = __ffma2_rn(make_float2(aa[u], aa[u]), make_float2(v.z, v.w), acc[u][1]);
          }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
          if (h0 + u < heads)
            store4(dst + (static_cast<size_t>(r) * heads + u) * kv_heads * D, make_float4(acc[u][0].x, acc[u][0].y, acc[u][1].x, acc[u][1].y));
      }
    }
    return;
  }
  for (int it = threadIdx.x; it < items; it += blockDim.x) {
    const int r = it / per_row, rest = it - r * per_row;
    const int h0 = rest / d4 * 4, d = (rest % d4) * 4;
    const float* qr = qs + r * row_q + d;
    float4 acc[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) acc[u] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int g = 0; g < per; ++g) {
      const float4 v = *reinterpret_cast<const float4*>(qr + g * D);
      const float4 a = *reinterpret_cast<const float4*>(ms + g * hp + h0);
      const float aa[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        acc[u].x = fmaf(aa[u], v.x, acc[u].x);
        acc[u].y = fmaf(aa[u], v.y, acc[u].y);
        acc[u].z = fmaf(aa[u], v.z, acc[u].z);
        acc[u].w = fmaf(aa[u], v.w, acc[u].w);
      }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (h0 + u >= heads) break;
      store4(out + ((static_cast<size_t>(m0 + r) * heads + h0 + u) * kv_heads + c) * D + d, acc[u]);
    }
  }
}

// Causal convolution per channel, then SiLU.  The inputs before the rows at hand come from a ring of `taps` rows per slot
// (position p of the sequence in row p % taps): one more than the convolution looks back, so that a decode step overwrites
// nothing it reads and may be run again.
// chunk: the rows are consecutive positions of one sequence, positions[0] on, with slot slots[0]; a CTA takes
// `rows_per` of them, the first CTA alone reads the ring (rows_per >= taps - 1) and, each column by the thread that has
// read it, writes it.  Otherwise every row is a sequence of its own.
// TAPS > 0: that many, weights and the window's rows in registers; 0: `taps`, every row read again for every tap.
template <typename T, int TAPS>
__global__ void __launch_bounds__(64)
conv_silu_kernel(const T* __restrict__ in, const T* __restrict__ w, int taps, T* __restrict__ ring,
                 const int* __restrict__ slots, const int* __restrict__ positions, int num_rows, int chunk, int rows_per,
                 int C, int num_slots, T* __restrict__ out, int* __restrict__ err) {
  grid_dep_wait();
  grid_dep_launch();
  const int col = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (col >= C) return;
  const int lo = blockIdx.x * rows_per, hi = min(num_rows, lo + rows_per);
  const int seq = chunk ? 0 : blockIdx.x;
  const int first = positions[seq];  // position of the sequence's first row at hand
  const int base = chunk ? 0 : lo;   // that row
  int slot = slots[seq];
  if (slot < 0 || slot >= num_slots || first < 0) {
    set_error(err, kErrDevBadBlockId);
    return;
  }
  T* hist = taps > 1 ? ring + static_cast<size_t>(slot) * taps * C + col : nullptr;
  if (TAPS > 1) {
    float w_r[TAPS > 1 ? TAPS : 1][8];
    Raw8<T> win[TAPS > 1 ? TAPS - 1 : 1];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load8<T>(w + static_cast<size_t>(j) * C + col, w_r[j]);
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j) {
      const int r = lo - (TAPS - 1 - j), pos = first + (r - base);
      if (pos < 0) win[j].zero();
      else if (r >= base) win[j].load(in + static_cast<size_t>(r) * C + col);
      else win[j].load(hist + static_cast<size_t>(pos % TAPS) * C);
    }
#pragma unroll 4
    for (int r = lo; r < hi; ++r) {
      Raw8<T> x;
      x.load(in + static_cast<size_t>(r) * C + col);
      float acc[8], f[8];
      x.get(f);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = 0.f;
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) {
        float a[8];
        win[j].get(a);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = fmaf(w_r[j][e], a[e], acc[e]);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = silu_as<T>(fmaf(w_r[TAPS > 0 ? TAPS - 1 : 0][e], f[e], acc[e]));
#pragma unroll
      for (int j = 0; j + 2 < TAPS; ++j) win[j] = win[j + 1];
      win[TAPS > 1 ? TAPS - 2 : 0] = x;
      store8<T>(out + static_cast<size_t>(r) * C + col, acc);
    }
  } else
#pragma unroll 2
  for (int r = lo; r < hi; ++r) {
    const int pos = first + (r - base);
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
#pragma unroll 4
    for (int j = 0; j < taps; ++j) {
      const int back = taps - 1 - j;
      if (pos - back < 0) continue;
      float a[8], b[8];
      if (r - back >= base) load8<T>(in + static_cast<size_t>(r - back) * C + col, a);
      else load8<T>(hist + static_cast<size_t>((pos - back) % taps) * C, a);
      load8<T>(w + static_cast<size_t>(j) * C + col, b);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = fmaf(b[e], a[e], acc[e]);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = silu_as<T>(acc[e]);
    store8<T>(out + static_cast<size_t>(r) * C + col, acc);
  }
  if (hist == nullptr || (chunk && blockIdx.x != 0)) return;
  const int end = chunk ? num_rows : lo + 1;
  for (int r = max(base, end - taps); r < end; ++r) {
    Raw8<T> v;
    v.load(in + static_cast<size_t>(r) * C + col);
    float f[8];
    v.get(f);
    store8<T>(hist + static_cast<size_t>((first + (r - base)) % taps) * C, f);
  }
}

// out = o / rms(o over the group) * w * gate * scale, o [M, groups, ldg] fp32 whose columns past `size` are zero.  LANES threads
// per (row, group): a warp (four to a block), or a block of 256 for long groups.  `shared_w`: one weight row for all groups.
template <typename T, int LANES>
__global__ void __launch_bounds__(LANES > 32 ? LANES : 128)
group_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ w, const T* __restrict__ gate, float eps,
                       int total, int groups, int size, int ldg, int shared_w, float scale, T* __restrict__ out, int out_ld) {
  __shared__ float part[LANES / 32];
  grid_dep_wait();
  grid_dep_launch();
  const int item = LANES > 32 ? blockIdx.x : blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x % LANES;
  if (item >= total) return;  // the whole warp or block
  const int m = item / groups, g = item - m * groups;
  const float* src = o + static_cast<size_t>(item) * ldg;
  float ss = 0.f;
#pragma unroll 4
  for (int c = lane * 4; c < ldg; c += LANES * 4) {
    const float4 v = *reinterpret_cast<const float4*>(src + c);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  ss = warp_sum(ss);
  if (LANES > 32) {
    if ((lane & 31) == 0) part[lane >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < LANES / 32; ++i) ss += part[i];
  }
  const float inv = scale / sqrtf(ss / static_cast<float>(size) + eps);
  const float* wg = w + (shared_w ? 0 : static_cast<size_t>(g) * ldg);
  const T* gt = gate + static_cast<size_t>(item) * ldg;
  T* dst = out + static_cast<size_t>(m) * out_ld + static_cast<size_t>(g) * ldg;
#pragma unroll 4
  for (int c = lane * 4; c < ldg; c += LANES * 4) {
    const float4 v = *reinterpret_cast<const float4*>(src + c), a = *reinterpret_cast<const float4*>(wg + c);
    const float g0 = to_f32<T>(gt[c]), g1 = to_f32<T>(gt[c + 1]), g2 = to_f32<T>(gt[c + 2]), g3 = to_f32<T>(gt[c + 3]);
    store4(dst + c, make_float4(v.x * inv * a.x * g0, v.y * inv * a.y * g1, v.z * inv * a.z * g2, v.w * inv * a.w * g3));
  }
}

template <typename T>
static int launch_residual_norm(float* x, const void* dense, const void* expert_rows, const int* row_of_pair,
                                const float* pair_weight, int top_k, const float* bias, const void* gate,
                                const float* weight, float eps, int rows, int width, int ld, int center, void* out,
                                cudaStream_t st) {
  const Pending<T> p{static_cast<const T*>(dense), static_cast<const T*>(expert_rows), row_of_pair, pair_weight, top_k, bias,
                     static_cast<const T*>(gate)};
  const int threads = (ld / 8 + 31) / 32 * 32;
#define B200_RNORM(CENTER, MAXT)                                                                                     \
  B200_CUDA(launch_overlapped(residual_norm_kernel<T, CENTER, MAXT>, dim3(rows), dim3(threads), 0, st, x, p, weight, eps, \
                              width, ld, static_cast<T*>(out)))
  if (threads <= 512) {
    if (center) B200_RNORM(true, 512);
    else B200_RNORM(false, 512);
  } else {
    if (center) B200_RNORM(true, 1024);
    else B200_RNORM(false, 1024);
  }
#undef B200_RNORM
  return 0;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_residual_norm(float* x, const void* delta, const void* expert_rows, const int32_t* row_of_pair,
                                  const float* pair_weight, int top_k, const float* bias, const void* gate,
                                  const float* weight, float eps, int num_rows, int width, int ld, int center, void* out,
                                  int dtype, void* stream) {
  B200_REQUIRE(x && weight && out, "residual_norm: null pointer");
  B200_REQUIRE(num_rows >= 0 && width > 0 && ld >= width && ld % 8 == 0 && ld <= 8192,
               "residual_norm: width %d (pitch %d, at most 8192)", width, ld);
  B200_REQUIRE(!(delta && expert_rows) && (!expert_rows || (row_of_pair && pair_weight && top_k > 0)),
               "residual_norm: rows of one kind, expert rows with their pairs");
  B200_REQUIRE(aligned16({x, delta, expert_rows, bias, gate, weight, out}), "residual_norm: buffers must be 16-byte aligned");
  B200_GLUE_DTYPE("residual_norm");
  if (num_rows == 0) return 0;
  return dtype == 0 ? launch_residual_norm<__nv_bfloat16>(x, delta, expert_rows, row_of_pair, pair_weight, top_k, bias, gate,
                                                          weight, eps, num_rows, width, ld, center, out, as_stream(stream))
                    : launch_residual_norm<float>(x, delta, expert_rows, row_of_pair, pair_weight, top_k, bias, gate, weight,
                                                  eps, num_rows, width, ld, center, out, as_stream(stream));
}

extern "C" int b200_mix_heads(const void* q, const float* mix, void* out, int num_rows, int heads, int kv_heads,
                              int head_dim, int dtype, void* stream) {
  B200_REQUIRE(q && mix && out, "mix_heads: null pointer");
  B200_REQUIRE(num_rows >= 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && kv_heads <= 65535 && head_dim > 0 &&
                   head_dim % 4 == 0,
               "mix_heads: %d heads over %d kv heads of %d", heads, kv_heads, head_dim);
  B200_REQUIRE(aligned16({q, out}), "mix_heads: buffers must be 16-byte aligned");
  const int per = heads / kv_heads;
  const size_t mix_bytes = static_cast<size_t>(per) * ((heads + 3) & ~3) * 4, row_bytes = static_cast<size_t>(per) * head_dim * 4;
  int rows_per = num_rows * kv_heads >= 4096 ? 8 : 1;  // many rows: the mixing matrix is fetched once for several
  while (rows_per > 1 && mix_bytes + rows_per * row_bytes > 64 * 1024) rows_per >>= 1;
  const size_t smem = mix_bytes + rows_per * row_bytes;
  B200_REQUIRE(smem <= 200 * 1024, "mix_heads: %d heads of %d per kv head do not fit", per, head_dim);
  B200_GLUE_DTYPE("mix_heads");
  if (num_rows == 0) return 0;
  const dim3 grid((num_rows + rows_per - 1) / rows_per, kv_heads);
  if (dtype == 0) {
    int rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&mix_heads_kernel<__nv_bfloat16>), 200 * 1024);
    if (rc) return rc;
    B200_CUDA(launch_overlapped(mix_heads_kernel<__nv_bfloat16>, grid, dim3(256), smem, as_stream(stream),
                                static_cast<const __nv_bfloat16*>(q), mix, static_cast<__nv_bfloat16*>(out), num_rows, rows_per, heads, kv_heads, head_dim));
  } else {
    int rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&mix_heads_kernel<float>), 200 * 1024);
    if (rc) return rc;
    B200_CUDA(launch_overlapped(mix_heads_kernel<float>, grid, dim3(256), smem, as_stream(stream), static_cast<const float*>(q), mix,
                                static_cast<float*>(out), num_rows, rows_per, heads, kv_heads, head_dim));
  }
  return 0;
}

extern "C" int b200_conv_silu(const void* in, const void* conv_w, int taps, void* ring, const int32_t* slots,
                              const int32_t* positions, int num_rows, int chunk, int channels, int num_slots, void* out,
                              void* status_word, int dtype, void* stream) {
  B200_REQUIRE(in && conv_w && slots && positions && out && in != out, "conv_silu: null pointer (or in place)");
  B200_REQUIRE(num_rows >= 0 && taps >= 1 && (taps == 1 || ring) && channels > 0 && channels % 8 == 0 && num_slots > 0,
               "conv_silu: %d rows, %d taps, %d channels", num_rows, taps, channels);
  B200_REQUIRE(aligned16({in, conv_w, ring, out}), "conv_silu: buffers must be 16-byte aligned");
  B200_GLUE_DTYPE("conv_silu");
  if (num_rows == 0) return 0;
  const int rows_per = chunk ? (taps - 1 > 8 ? taps - 1 : 8) : 1;
  const dim3 grid((num_rows + rows_per - 1) / rows_per, (channels / 8 + 63) / 64);
  int* err = static_cast<int*>(status_word);
#define B200_CONV(T, TAPS)                                                                                                     \
  B200_CUDA(launch_overlapped(conv_silu_kernel<T, TAPS>, grid, dim3(64), 0, as_stream(stream), static_cast<const T*>(in),      \
                              static_cast<const T*>(conv_w), taps, static_cast<T*>(ring), slots, positions, num_rows, chunk,   \
                              rows_per, channels, num_slots, static_cast<T*>(out), err))
  if (dtype == 0) {
    if (taps == 2) B200_CONV(__nv_bfloat16, 2);
    else if (taps == 3) B200_CONV(__nv_bfloat16, 3);
    else if (taps == 4) B200_CONV(__nv_bfloat16, 4);
    else B200_CONV(__nv_bfloat16, 0);
  } else {
    B200_CONV(float, 0);
  }
#undef B200_CONV
  return 0;
}

extern "C" int b200_group_norm_gate(const float* o, const float* weight, const void* gate, float eps, int num_rows,
                                    int groups, int size, int group_ld, int shared_weight, float scale, void* out,
                                    int out_ld, int dtype, void* stream) {
  B200_REQUIRE(o && weight && gate && out, "group_norm_gate: null pointer");
  B200_REQUIRE(num_rows >= 0 && groups > 0 && size > 0 && group_ld >= size && group_ld % 4 == 0 && out_ld % 4 == 0 &&
                   out_ld >= groups * group_ld,
               "group_norm_gate: %d groups of %d (pitch %d)", groups, size, group_ld);
  B200_REQUIRE(aligned16({o, weight}) && (reinterpret_cast<uintptr_t>(out) & 7) == 0 &&
                   (dtype == 0 || (reinterpret_cast<uintptr_t>(out) & 15) == 0),
               "group_norm_gate: buffers must be aligned");
  B200_REQUIRE(static_cast<long long>(num_rows) * groups < (1ll << 31), "group_norm_gate: too many rows");
  B200_GLUE_DTYPE("group_norm_gate");
  if (num_rows == 0) return 0;
  const int total = num_rows * groups;
#define B200_GROUP_NORM(T, LANES)                                                                                     \
  B200_CUDA(launch_overlapped(group_norm_gate_kernel<T, LANES>, dim3(LANES > 32 ? total : (total + 3) / 4),            \
                              dim3(LANES > 32 ? LANES : 128), 0, as_stream(stream), o, weight, static_cast<const T*>(gate), eps, \
                              total, groups, size, group_ld, shared_weight, scale, static_cast<T*>(out), out_ld))
  if (dtype == 0 && group_ld >= 1024) B200_GROUP_NORM(__nv_bfloat16, 256);
  else if (dtype == 0) B200_GROUP_NORM(__nv_bfloat16, 32);
  else if (group_ld >= 1024) B200_GROUP_NORM(float, 256);
  else B200_GROUP_NORM(float, 32);
#undef B200_GROUP_NORM
  return 0;
}
