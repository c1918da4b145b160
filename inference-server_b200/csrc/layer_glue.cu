// Small kernels between the matrix products of the layer-list decoders (engine: layered.py): token + sinusoid
// embedding, residual add + grouped RMSNorm, the short causal convolution ahead of a mixer, the latents' norm and page
// write, and the unfused forms that the fp32 engine uses.  The residual stream is fp32 throughout, statistics and
// convolutions are fp32; T is the type of the activations between kernels (bf16 or fp32).
//
// The convolution's history lives in the pages, beside the K/V or latents of the same tokens: per layer
// hist [num_blocks, min(taps, page), ld], position p of a sequence in its page p / page, slot (p % page) % rows.
// The taps - 1 rows before any position are then always to be found: each is among the last `rows` written in its page.
// One row more than the convolution looks back makes a step repeatable: writing position p overwrites none of the rows
// that p itself reads (a CUDA graph's warm-up runs the same step several times).
// A sequence's state is taken, moved and given back with its pages, and there is no slot to manage.

#include "glue.cuh"

namespace b200 {

constexpr int kGlueMaxSegs = 8;
constexpr int kFastTaps = 5;  // convolutions of up to this many taps keep their rows in registers

template <typename T>
__global__ void embed_sinusoid_kernel(const long long* __restrict__ tokens, const int* __restrict__ positions,
                                      const T* __restrict__ embed, const float* __restrict__ lo,
                                      const float* __restrict__ hi, float* __restrict__ x, int* __restrict__ err,
                                      int width, int ld, int vocab, int n_hi) {
  grid_dep_wait();
  grid_dep_launch();
  const int m = blockIdx.x;
  long long tok = tokens[m];
  int pos = positions[m];
  if (tok < 0 || tok >= vocab || pos < 0 || pos >= n_hi * 64) {
    if (threadIdx.x == 0) set_error(err, kErrDevBadCtxLen);
    tok = 0;
    pos = 0;
  }
  const T* e = embed + static_cast<size_t>(tok) * ld;
  float* o = x + static_cast<size_t>(m) * ld;
  if (lo == nullptr) {  // no sinusoid
    for (int c = threadIdx.x * 2; c < ld; c += blockDim.x * 2)
      *reinterpret_cast<float2*>(o + c) = make_float2(c < width ? to_f32<T>(e[c]) : 0.f, c + 1 < width ? to_f32<T>(e[c + 1]) : 0.f);
    return;
  }
  const float* l = lo + static_cast<size_t>(pos & 63) * ld;
  const float* h = hi + static_cast<size_t>(pos >> 6) * ld;
  for (int c = threadIdx.x * 2; c < ld; c += blockDim.x * 2) {
    const float2 a = *reinterpret_cast<const float2*>(h + c), b = *reinterpret_cast<const float2*>(l + c);
    float2 r;  // sin(a + b), cos(a + b)
    r.x = c < width ? to_f32<T>(e[c]) + fmaf(a.x, b.y, a.y * b.x) : 0.f;
    r.y = c + 1 < width ? to_f32<T>(e[c + 1]) + fmaf(a.y, b.y, -(a.x * b.x)) : 0.f;
    *reinterpret_cast<float2*>(o + c) = r;
  }
}

// One CTA per row, 8 columns per thread.  WIDE: a group's width is a multiple of 256, so every warp lies in one group.
template <typename T, bool WIDE, int MAXT>
__global__ void __launch_bounds__(MAXT)
group_rmsnorm_kernel(float* __restrict__ x, const T* __restrict__ delta, const T* __restrict__ weight,
                                     float eps, int width, int ld, int groups, T* __restrict__ out,
                                     const T* __restrict__ conv_w, int taps, T* __restrict__ hist,
                                     const int* __restrict__ positions, const int* __restrict__ block_table, PageMap pm) {
  grid_dep_wait();
  grid_dep_launch();
  extern __shared__ float sm[];
  const int m = blockIdx.x, col = threadIdx.x * 8;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool in = col < ld;
  const size_t at = static_cast<size_t>(m) * ld + col;
  const int gs = width / groups;
  float f[8], w[8], acc[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) f[j] = w[j] = acc[j] = 0.f;
  // the convolution's earlier rows do not depend on this row: their pages are looked up first, the rows themselves asked
  // for before the statistics
  int pos = 0, page = -1, before = -1, rows = 0;
  const int* table_row = nullptr;
  if (taps > 0) {
    pos = positions[m];
    table_row = block_table + static_cast<size_t>(m) * pm.max_pages;
    page = page_of(pm, table_row, pos);
    if (pos >= pm.page) before = page_of(pm, table_row, pos - pm.page);
    rows = taps > 1 ? min(taps, pm.page) : 0;
  }
  if (in) {
    load8<float>(x + at, f);
    load8<T>(weight + col, w);
    if (delta != nullptr) {
      float d[8];
      load8<T>(delta + at, d);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] += d[j];
      store8<float>(x + at, f);
    }
  }
  float wlast[8];
  if (taps > 0) {
    if (in && page >= 0) {
      load8<T>(conv_w + static_cast<size_t>(taps - 1) * ld + col, wlast);
    }
    if (taps <= kFastTaps && taps - 1 <= pm.page) {
      // the earlier rows lie in this page and the one before: all rows and weights are in flight together
      const int slot0 = pos % pm.page;
      Raw8<T> hv[kFastTaps - 1], cw[kFastTaps - 1];
#pragma unroll
      for (int j = 0; j < kFastTaps - 1; ++j) {
        const int s = pos - taps + 1 + j;
        const int back = slot0 - (taps - 1 - j);  // slot in this page, negative: in the page before
        const int pg = back >= 0 ? page : before;
        hv[j].zero();
        cw[j].zero();
        if (in && j + 1 < taps && s >= 0 && pg >= 0) {
          hv[j].load(hist + (static_cast<size_t>(pg) * rows + (back >= 0 ? back : back + pm.page) % rows) * ld + col);
          cw[j].load(conv_w + static_cast<size_t>(j) * ld + col);
        }
      }
#pragma unroll
      for (int j = 0; j < kFastTaps - 1; ++j) {
        float a[8], b[8];
        hv[j].get(a);
        cw[j].get(b);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = fmaf(b[e], a[e], acc[e]);
      }
    } else if (in && page >= 0) {
      for (int j = 0; j + 1 < taps; ++j) {
        const int s = pos - taps + 1 + j;
        if (s < 0) continue;
        const int pg = page_of(pm, table_row, s);
        if (pg < 0) continue;
        float hv[8], cw[8];
        load8<T>(hist + (static_cast<size_t>(pg) * rows + (s % pm.page) % rows) * ld + col, hv);
        load8<T>(conv_w + static_cast<size_t>(j) * ld + col, cw);
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = fmaf(cw[e], hv[e], acc[e]);
      }
    }
  }
  float inv[8];
  if (WIDE) {
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
    ss = warp_sum(ss);
    if (lane == 0) sm[warp] = ss;
    __syncthreads();
    const int per = gs >> 8, g = warp / per;  // warps per group
    float t = 0.f;
    for (int i = 0; i < per; ++i) t += sm[g * per + i];
    const float r = 1.f / sqrtf(t / static_cast<float>(gs) + eps);
#pragma unroll
    for (int j = 0; j < 8; ++j) inv[j] = r;
  } else {
    float* sq = sm;
    float* gi = sm + ld;
#pragma unroll
    for (int j = 0; j < 8; ++j) inv[j] = f[j] * f[j];
    if (in) store8<float>(sq + col, inv);
    __syncthreads();
    for (int g = warp; g < groups; g += blockDim.x >> 5) {
      float t = 0.f;
      for (int i = lane; i < gs; i += 32) t += sq[g * gs + i];
      t = warp_sum(t);
      if (lane == 0) gi[g] = 1.f / sqrtf(t / static_cast<float>(gs) + eps);
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < 8; ++j) inv[j] = col + j < width ? gi[(col + j) / gs] : 0.f;
  }
  if (!in) return;
  float y[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) y[j] = f[j] * inv[j] * w[j];
  if (taps > 0) {
    if (page < 0) return;
#pragma unroll
    for (int j = 0; j < 8; ++j) y[j] = round_to<T>(y[j]);
    if (rows > 0) store8<T>(hist + (static_cast<size_t>(page) * rows + (pos % pm.page) % rows) * ld + col, y);
#pragma unroll
    for (int j = 0; j < 8; ++j) y[j] = y[j] + fmaf(wlast[j], y[j], acc[j]);
  }
  store8<T>(out + at, y);
}

// Rows of one page of the sequence per CTA (blockIdx.x), 8 columns per thread.  The only rows read from the history
// lie before the chunk; a page's history is written by the CTA of that page alone, each column by the thread that has
// read it, so the first page's writes come after its reads.  Reads further back are of pages that nobody writes.
// TAPS > 0: that many, the rows of the window kept in registers; 0: `taps`, each row read again for every tap.
template <typename T, int TAPS>
__global__ void __launch_bounds__(64)
short_conv_kernel(const T* __restrict__ h, const T* __restrict__ conv_w, int taps, T* __restrict__ hist,
                  const int* __restrict__ table_row, int num_rows, int first_pos, int ld, T* __restrict__ out,
                  PageMap pm) {
  grid_dep_wait();
  grid_dep_launch();
  const int col = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (col >= ld) return;
  const int pg0 = first_pos / pm.page + static_cast<int>(blockIdx.x);
  const int lo = max(first_pos, pg0 * pm.page), hi = min(first_pos + num_rows, (pg0 + 1) * pm.page);
  const int rows = taps > 1 ? min(taps, pm.page) : 0;
  if (TAPS > 1) {
    float w[TAPS > 1 ? TAPS : 1][8], win[TAPS > 1 ? TAPS - 1 : 1][8];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load8<T>(conv_w + static_cast<size_t>(j) * ld + col, w[j]);
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j) {
      const int s = lo - TAPS + 1 + j;
#pragma unroll
      for (int e = 0; e < 8; ++e) win[j][e] = 0.f;
      if (s >= first_pos) {
        load8<T>(h + static_cast<size_t>(s - first_pos) * ld + col, win[j]);
      } else if (s >= 0) {
        const int pg = page_of(pm, table_row, s);
        if (pg >= 0) load8<T>(hist + (static_cast<size_t>(pg) * rows + (s % pm.page) % rows) * ld + col, win[j]);
      }
    }
#pragma unroll 4
    for (int p = lo; p < hi; ++p) {
      float hv[8], acc[8];
      load8<T>(h + static_cast<size_t>(p - first_pos) * ld + col, hv);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = 0.f;
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = fmaf(w[j][e], win[j][e], acc[e]);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = fmaf(w[TAPS > 0 ? TAPS - 1 : 0][e], hv[e], acc[e]) + hv[e];
#pragma unroll
      for (int j = 0; j + 2 < TAPS; ++j)
#pragma unroll
        for (int e = 0; e < 8; ++e) win[j][e] = win[j + 1][e];
#pragma unroll
      for (int e = 0; e < 8; ++e) win[TAPS > 1 ? TAPS - 2 : 0][e] = hv[e];
      store8<T>(out + static_cast<size_t>(p - first_pos) * ld + col, acc);
    }
  } else
#pragma unroll 2
  for (int p = lo; p < hi; ++p) {
    float acc[8], hv[8], cw[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
    for (int j = 0; j < taps; ++j) {
      const int s = p - taps + 1 + j;
      if (s < 0) continue;
      if (s >= first_pos) {
        load8<T>(h + static_cast<size_t>(s - first_pos) * ld + col, hv);
      } else {
        const int pg = page_of(pm, table_row, s);
        if (pg < 0) continue;
        load8<T>(hist + (static_cast<size_t>(pg) * rows + (s % pm.page) % rows) * ld + col, hv);
      }
      load8<T>(conv_w + static_cast<size_t>(j) * ld + col, cw);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = fmaf(cw[e], hv[e], acc[e]);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] += hv[e];  // hv is row p itself after the last tap
    store8<T>(out + static_cast<size_t>(p - first_pos) * ld + col, acc);
  }
  const int id = rows > 0 ? page_of(pm, table_row, lo) : -1;
  if (id < 0) return;
  for (int p = max(lo, hi - rows); p < hi; ++p) {
    float hv[8];
    load8<T>(h + static_cast<size_t>(p - first_pos) * ld + col, hv);
    store8<T>(hist + (static_cast<size_t>(id) * rows + (p % pm.page) % rows) * ld + col, hv);
  }
}

// One warp per row.
template <typename T>
__global__ void __launch_bounds__(128)
latent_norm_append_kernel(const float* __restrict__ raw, const T* __restrict__ weight, float eps, int num_rows, int rank,
                          int ld, T* __restrict__ c_pool, const int* __restrict__ positions,
                          const int* __restrict__ block_table, PageMap pm) {
  grid_dep_wait();
  grid_dep_launch();
  const int m = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (m >= num_rows) return;
  const int pos = positions[m];
  const float* r = raw + static_cast<size_t>(m) * ld;
  const int page = page_of(pm, block_table + static_cast<size_t>(m) * pm.max_pages, pos);
  float ss = 0.f;
  for (int c = lane * 4; c < ld; c += 128) {  // columns past rank are zero
    const float4 v = *reinterpret_cast<const float4*>(r + c);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(rank) + eps);
  if (page < 0) return;
  T* dst = c_pool + (static_cast<size_t>(page) * pm.page + pos % pm.page) * ld;
  for (int c = lane; c < ld; c += 32) dst[c] = from_f32<T>(r[c] * inv * to_f32<T>(weight[c]));
}

// 16 bytes per thread.
__global__ void gather_pages_kernel(const uint4* __restrict__ pool, const int* __restrict__ table_row,
                                    uint4* __restrict__ out, int num_tokens, int vec, PageMap pm) {
  grid_dep_wait();
  grid_dep_launch();
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  const int tok = static_cast<int>(i / vec), v = static_cast<int>(i - static_cast<long long>(tok) * vec);
  if (tok >= num_tokens) return;
  const int id = page_of(pm, table_row, tok);
  out[i] = id < 0 ? make_uint4(0u, 0u, 0u, 0u) : pool[(static_cast<size_t>(id) * pm.page + tok % pm.page) * vec + v];
}

struct GlueSegs {
  int end[kGlueMaxSegs], kind[kGlueMaxSegs], act[kGlueMaxSegs], heads[kGlueMaxSegs], dim[kGlueMaxSegs];
  void* ptr[kGlueMaxSegs];
  int count;
};

template <typename T>
__global__ void split_store_kernel(const float* __restrict__ y, const float* __restrict__ col_scale,
                                   const float* __restrict__ col_bias, GlueSegs segs,
                                   const int* __restrict__ positions, const int* __restrict__ block_table, PageMap pm) {
  const int m = blockIdx.x, total = segs.end[segs.count - 1];
  const int pos = positions != nullptr ? positions[m] : m;
  int id = -2;  // looked up when a page segment is met
  for (int n = threadIdx.x; n < total; n += blockDim.x) {
    float v = y[static_cast<size_t>(m) * total + n];
    if (col_scale != nullptr) v *= col_scale[n];
    if (col_bias != nullptr) v += col_bias[n];
    int s = 0, begin = 0;
    while (n >= segs.end[s]) begin = segs.end[s++];
    if (segs.act[s] == 1) v = silu_of(v);
    else if (segs.act[s] == 2) v = sigmoid_of(v);
    const int local = n - begin, wd = segs.end[s] - begin;
    if (segs.kind[s] == 0) {
      static_cast<T*>(segs.ptr[s])[static_cast<size_t>(m) * wd + local] = from_f32<T>(v);
    } else if (segs.kind[s] == 1) {
      static_cast<float*>(segs.ptr[s])[static_cast<size_t>(m) * wd + local] = v;
    } else {
      if (id == -2) {
        if (block_table != nullptr) id = page_of(pm, block_table + static_cast<size_t>(m) * pm.max_pages, pos);
        else id = pos >= 0 && pos / pm.page < pm.num_blocks ? pos / pm.page : -1;
      }
      const int head = local / segs.dim[s], d = local - head * segs.dim[s];
      if (id >= 0)
        static_cast<T*>(segs.ptr[s])[((static_cast<size_t>(id) * segs.heads[s] + head) * pm.page + pos % pm.page) * segs.dim[s] + d] =
            from_f32<T>(v);
    }
  }
}

// gate_up [rows, 2 * inter], gate and up columns in alternating blocks of 128.
template <typename T>
__global__ void clamped_glu_kernel(const T* __restrict__ gu, T* __restrict__ out, long long total, int inter, float limit,
                                   float alpha, float shift) {
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const long long m = i / inter;
  const int n = static_cast<int>(i - m * inter);
  const T* row = gu + m * 2 * inter + (n / 128) * 256 + n % 128;
  out[i] = from_f32<T>(clamped_glu(to_f32<T>(row[0]), to_f32<T>(row[128]), limit, alpha, shift));
}

__global__ void __launch_bounds__(256)
argmax_rows_kernel(const float* __restrict__ logits, long long* __restrict__ out, int n) {
  __shared__ float bv_sm[8];
  __shared__ int bi_sm[8];
  const float* r = logits + static_cast<size_t>(blockIdx.x) * n;
  float bv = -INFINITY;
  int bi = 0x7fffffff;
  for (int i = threadIdx.x; i < n; i += 256) {
    const float v = r[i];
    if (v > bv || bi == 0x7fffffff) {
      bv = v;
      bi = i;
    }
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ov > bv || (ov == bv && oi < bi)) {
      bv = ov;
      bi = oi;
    }
  }
  if (lane == 0) {
    bv_sm[warp] = bv;
    bi_sm[warp] = bi;
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int w = 1; w < 8; ++w)
      if (bv_sm[w] > bv || (bv_sm[w] == bv && bi_sm[w] < bi)) {
        bv = bv_sm[w];
        bi = bi_sm[w];
      }
    out[blockIdx.x] = bi == 0x7fffffff ? 0 : bi;
  }
}

// fp32 product, 64 x 64 tile per CTA, 4 x 4 per thread, K in steps of 16 (K a multiple of 4, zero fill past it).
// Every element is summed over k in the same order whatever the shape.
__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, float* __restrict__ y, int M, int N, int K,
                int x_step, int w_step, int y_step, int ldx, int ldy, const MoeTile* __restrict__ tiles,
                const int* __restrict__ num_tiles, int num_experts) {
  __shared__ float xs[16][64 + 4], ws[16][64 + 4];
  int g = blockIdx.z, m0 = blockIdx.y * 64;
  const int n0 = blockIdx.x * 64;
  if (tiles != nullptr) {  // rows sorted by expert: blockIdx.y counts tiles of at most 64 rows of one expert
    if (static_cast<int>(blockIdx.y) >= *num_tiles) return;
    const MoeTile t = tiles[blockIdx.y];
    if (t.expert < 0 || t.expert >= num_experts || t.row0 < 0 || t.rows < 0 || t.rows > 64 || t.row0 + t.rows > M) return;
    g = t.expert;
    m0 = t.row0;
    M = t.row0 + t.rows;
    x_step = y_step = 0;
  }
  const int tid = threadIdx.x, r = tid >> 2, kq = (tid & 3) * 4;
  const int ty = tid >> 4, tx = tid & 15;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += 16) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
    if (k0 + kq < K) {
      if (m0 + r < M) a = *reinterpret_cast<const float4*>(x + static_cast<size_t>(m0 + r) * ldx + g * x_step + k0 + kq);
      if (n0 + r < N) b = *reinterpret_cast<const float4*>(w + (static_cast<size_t>(g) * w_step + n0 + r) * K + k0 + kq);
    }
    __syncthreads();
    xs[kq][r] = a.x; xs[kq + 1][r] = a.y; xs[kq + 2][r] = a.z; xs[kq + 3][r] = a.w;
    ws[kq][r] = b.x; ws[kq + 1][r] = b.y; ws[kq + 2][r] = b.z; ws[kq + 3][r] = b.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float4 bv = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float aa[4] = {av.x, av.y, av.z, av.w}, bb[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(aa[i], bb[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) y[static_cast<size_t>(m) * ldy + g * y_step + n] = acc[i][j];
    }
  }
}

template <typename T>
static int launch_group_rmsnorm(float* x, const void* delta, const void* weight, float eps, int rows, int width, int ld,
                                int groups, void* out, const void* conv_w, int taps, void* hist, const int* positions,
                                const int* block_table, const PageMap& pm, cudaStream_t st) {
  const int threads = (ld / 8 + 31) / 32 * 32;
  const bool wide = (width / groups) % 256 == 0;
  const size_t smem = wide ? 32 * 4 : static_cast<size_t>(ld + groups) * 4;
#define B200_NORM_ARGS                                                                                              \
  x, static_cast<const T*>(delta), static_cast<const T*>(weight), eps, width, ld, groups, static_cast<T*>(out),      \
      static_cast<const T*>(conv_w), taps, static_cast<T*>(hist), positions, block_table, pm
  if (threads <= 512) {
    if (wide)
      B200_CUDA(launch_overlapped(group_rmsnorm_kernel<T, true, 512>, dim3(rows), dim3(threads), smem, st, B200_NORM_ARGS));
    else
      B200_CUDA(launch_overlapped(group_rmsnorm_kernel<T, false, 512>, dim3(rows), dim3(threads), smem, st, B200_NORM_ARGS));
  } else if (wide) {
    B200_CUDA(launch_overlapped(group_rmsnorm_kernel<T, true, 1024>, dim3(rows), dim3(threads), smem, st, B200_NORM_ARGS));
  } else {
    B200_CUDA(launch_overlapped(group_rmsnorm_kernel<T, false, 1024>, dim3(rows), dim3(threads), smem, st, B200_NORM_ARGS));
  }
#undef B200_NORM_ARGS
  return 0;
}

template <typename T>
static int launch_short_conv(const void* h, const void* conv_w, int taps, void* hist, const int* table_row, int rows,
                             int first_pos, int ld, void* out, const PageMap& pm, dim3 grid, cudaStream_t st) {
#define B200_CONV_CASE(TAPS)                                                                                             \
  B200_CUDA(launch_overlapped(short_conv_kernel<T, TAPS>, grid, dim3(64), 0, st, static_cast<const T*>(h),               \
                              static_cast<const T*>(conv_w), taps, static_cast<T*>(hist), table_row, rows, first_pos, ld, \
                              static_cast<T*>(out), pm))
  switch (taps) {
    case 2: B200_CONV_CASE(2); break;
    case 3: B200_CONV_CASE(3); break;
    case 4: B200_CONV_CASE(4); break;
    default: B200_CONV_CASE(0); break;
  }
#undef B200_CONV_CASE
  return 0;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_embed_sinusoid(const int64_t* tokens, const int32_t* positions, const void* embed, const float* lo,
                                   const float* hi, float* x, void* status_word, int num_rows, int width, int ld,
                                   int vocab, int n_hi, int dtype, void* stream) {
  B200_REQUIRE(tokens && positions && embed && (lo != nullptr) == (hi != nullptr) && x, "embed_sinusoid: null pointer");
  B200_REQUIRE(num_rows >= 0 && width > 0 && ld >= width && ld % 8 == 0 && vocab > 0 && n_hi > 0,
               "embed_sinusoid: rows %d, width %d, pitch %d", num_rows, width, ld);
  B200_REQUIRE(aligned16({lo, hi, x}), "embed_sinusoid: tables and x must be 16-byte aligned");
  B200_GLUE_DTYPE("embed_sinusoid");
  if (num_rows == 0) return 0;
  const int threads = ld / 2 >= 256 ? 256 : (ld / 2 + 31) / 32 * 32;
  const long long* tk = reinterpret_cast<const long long*>(tokens);
  int* err = static_cast<int*>(status_word);
  if (dtype == 0)
    B200_CUDA(launch_overlapped(embed_sinusoid_kernel<__nv_bfloat16>, dim3(num_rows), dim3(threads), 0, as_stream(stream),
                                tk, positions, static_cast<const __nv_bfloat16*>(embed), lo, hi, x, err, width, ld, vocab,
                                n_hi));
  else
    B200_CUDA(launch_overlapped(embed_sinusoid_kernel<float>, dim3(num_rows), dim3(threads), 0, as_stream(stream), tk,
                                positions, static_cast<const float*>(embed), lo, hi, x, err, width, ld, vocab, n_hi));
  return 0;
}

extern "C" int b200_group_rmsnorm(float* x, const void* delta, const void* weight, float eps, int num_rows, int width,
                                  int ld, int groups, void* out, const void* conv_w, int taps, void* hist,
                                  const int32_t* positions, const int32_t* block_table, int page_size, int num_blocks,
                                  int max_pages_per_seq, void* status_word, int dtype, void* stream) {
  B200_REQUIRE(x && weight && out, "group_rmsnorm: null pointer");
  B200_REQUIRE(num_rows >= 0 && width > 0 && ld >= width && ld % 8 == 0 && ld <= 8192 && groups > 0 && width % groups == 0,
               "group_rmsnorm: width %d (pitch %d, at most 8192) in %d groups", width, ld, groups);
  B200_REQUIRE(taps >= 0 && (taps == 0 || (conv_w && positions && block_table && page_size > 0 && num_blocks > 0 &&
                                           max_pages_per_seq > 0 && (taps == 1 || hist))),
               "group_rmsnorm: the convolution needs weights, positions, pages and a history");
  B200_REQUIRE(aligned16({x, delta, weight, out, conv_w, hist}), "group_rmsnorm: buffers must be 16-byte aligned");
  B200_GLUE_DTYPE("group_rmsnorm");
  if (num_rows == 0) return 0;
  const PageMap pm{page_size, num_blocks, max_pages_per_seq, static_cast<int*>(status_word)};
  if (dtype == 0)
    return launch_group_rmsnorm<__nv_bfloat16>(x, delta, weight, eps, num_rows, width, ld, groups, out, conv_w, taps, hist,
                                               positions, block_table, pm, as_stream(stream));
  return launch_group_rmsnorm<float>(x, delta, weight, eps, num_rows, width, ld, groups, out, conv_w, taps, hist, positions,
                                     block_table, pm, as_stream(stream));
}

extern "C" int b200_short_conv(const void* h, const void* conv_w, int taps, void* hist, const int32_t* block_table_row,
                               int num_rows, int first_position, int ld, void* out, int page_size, int num_blocks,
                               int max_pages_per_seq, void* status_word, int dtype, void* stream) {
  B200_REQUIRE(h && conv_w && block_table_row && out && h != out, "short_conv: null pointer (or in place)");
  B200_REQUIRE(num_rows > 0 && first_position >= 0 && taps >= 1 && (taps == 1 || hist) && ld > 0 && ld % 8 == 0 &&
                   page_size > 0 && num_blocks > 0 && max_pages_per_seq > 0,
               "short_conv: rows %d from %d, %d taps, pitch %d", num_rows, first_position, taps, ld);
  B200_REQUIRE(first_position + num_rows <= max_pages_per_seq * page_size, "short_conv: positions up to %d do not fit %d pages",
               first_position + num_rows, max_pages_per_seq);
  B200_REQUIRE(aligned16({h, conv_w, hist, out}), "short_conv: buffers must be 16-byte aligned");
  B200_GLUE_DTYPE("short_conv");
  const PageMap pm{page_size, num_blocks, max_pages_per_seq, static_cast<int*>(status_word)};
  const int pages = (first_position + num_rows - 1) / page_size - first_position / page_size + 1;
  const dim3 grid(pages, (ld / 8 + 63) / 64);
  if (dtype == 0)
    return launch_short_conv<__nv_bfloat16>(h, conv_w, taps, hist, block_table_row, num_rows, first_position, ld, out, pm, grid,
                                            as_stream(stream));
  return launch_short_conv<float>(h, conv_w, taps, hist, block_table_row, num_rows, first_position, ld, out, pm, grid,
                                  as_stream(stream));
}

extern "C" int b200_latent_norm_append(const float* raw, const void* weight, float eps, int num_rows, int rank, int ld,
                                       void* c_pool, const int32_t* positions, const int32_t* block_table, int page_size,
                                       int num_blocks, int max_pages_per_seq, void* status_word, int dtype, void* stream) {
  B200_REQUIRE(raw && weight && c_pool && positions && block_table, "latent_norm_append: null pointer");
  B200_REQUIRE(num_rows >= 0 && rank > 0 && ld >= rank && ld % 4 == 0 && page_size > 0 && num_blocks > 0 &&
                   max_pages_per_seq > 0,
               "latent_norm_append: rank %d, pitch %d", rank, ld);
  B200_REQUIRE(aligned16({raw, weight, c_pool}), "latent_norm_append: buffers must be 16-byte aligned");
  B200_GLUE_DTYPE("latent_norm_append");
  if (num_rows == 0) return 0;
  const PageMap pm{page_size, num_blocks, max_pages_per_seq, static_cast<int*>(status_word)};
  const dim3 grid((num_rows + 3) / 4);
  if (dtype == 0)
    B200_CUDA(launch_overlapped(latent_norm_append_kernel<__nv_bfloat16>, grid, dim3(128), 0, as_stream(stream), raw,
                                static_cast<const __nv_bfloat16*>(weight), eps, num_rows, rank, ld,
                                static_cast<__nv_bfloat16*>(c_pool), positions, block_table, pm));
  else
    B200_CUDA(launch_overlapped(latent_norm_append_kernel<float>, grid, dim3(128), 0, as_stream(stream), raw,
                                static_cast<const float*>(weight), eps, num_rows, rank, ld, static_cast<float*>(c_pool),
                                positions, block_table, pm));
  return 0;
}

extern "C" int b200_gather_pages(const void* c_pool, const int32_t* block_table_row, void* out, int num_tokens, int ld,
                                 int page_size, int num_blocks, int max_pages_per_seq, void* status_word, int dtype,
                                 void* stream) {
  B200_REQUIRE(c_pool && block_table_row && out, "gather_pages: null pointer");
  B200_REQUIRE(num_tokens >= 0 && ld > 0 && ld % 8 == 0 && page_size > 0 && num_blocks > 0 && max_pages_per_seq > 0 &&
                   num_tokens <= max_pages_per_seq * page_size,
               "gather_pages: %d tokens of pitch %d", num_tokens, ld);
  B200_REQUIRE(aligned16({c_pool, out}), "gather_pages: buffers must be 16-byte aligned");
  B200_GLUE_DTYPE("gather_pages");
  if (num_tokens == 0) return 0;
  const PageMap pm{page_size, num_blocks, max_pages_per_seq, static_cast<int*>(status_word)};
  const int vec = ld * (dtype == 0 ? 2 : 4) / 16;
  const long long total = static_cast<long long>(num_tokens) * vec;
  B200_CUDA(launch_overlapped(gather_pages_kernel, dim3(static_cast<unsigned>((total + 255) / 256)), dim3(256), 0,
                              as_stream(stream), static_cast<const uint4*>(c_pool), block_table_row,
                              static_cast<uint4*>(out), num_tokens, vec, pm));
  return 0;
}

extern "C" int b200_split_store(const float* y, const float* col_scale, const float* col_bias, const int32_t* seg_end,
                                const int32_t* seg_kind, const int32_t* seg_act, const int32_t* seg_heads, const int32_t* seg_dim, void* const* seg_ptr, int num_segs,
                                const int32_t* positions, const int32_t* block_table, void* status_word, int num_rows,
                                int page_size, int num_blocks, int max_pages_per_seq, int dtype, void* stream) {
  B200_REQUIRE(y && seg_end && seg_kind && seg_heads && seg_dim && seg_ptr && num_segs >= 1 && num_segs <= kGlueMaxSegs,
               "split_store: 1 to %d segments", kGlueMaxSegs);
  GlueSegs s{};
  s.count = num_segs;
  int begin = 0;
  for (int i = 0; i < num_segs; ++i) {
    B200_REQUIRE(seg_end[i] > begin && seg_ptr[i] && seg_kind[i] >= 0 && seg_kind[i] <= 2, "split_store: segment %d", i);
    if (seg_kind[i] == 2)
      B200_REQUIRE(seg_heads[i] > 0 && seg_dim[i] > 0 && seg_heads[i] * seg_dim[i] == seg_end[i] - begin && page_size > 0 &&
                       num_blocks > 0 && max_pages_per_seq > 0,
                   "split_store: page segment %d does not match its pool", i);
    s.end[i] = seg_end[i];
    s.kind[i] = seg_kind[i];
    s.act[i] = seg_act ? seg_act[i] : 0;
    s.heads[i] = seg_heads[i];
    s.dim[i] = seg_dim[i];
    s.ptr[i] = seg_ptr[i];
    begin = seg_end[i];
  }
  B200_GLUE_DTYPE("split_store");
  if (num_rows <= 0) return 0;
  const PageMap pm{page_size, num_blocks, max_pages_per_seq, static_cast<int*>(status_word)};
  if (dtype == 0)
    split_store_kernel<__nv_bfloat16><<<num_rows, 256, 0, as_stream(stream)>>>(y, col_scale, col_bias, s, positions, block_table, pm);
  else
    split_store_kernel<float><<<num_rows, 256, 0, as_stream(stream)>>>(y, col_scale, col_bias, s, positions, block_table, pm);
  B200_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int b200_clamped_glu(const void* gate_up, void* out, int num_rows, int inter, float limit, float alpha, float shift,
                                int dtype, void* stream) {
  B200_REQUIRE(gate_up && out && num_rows >= 0 && inter > 0 && inter % 128 == 0,
               "clamped_glu: %d rows of %d inner features (a multiple of 128)", num_rows, inter);
  B200_GLUE_DTYPE("clamped_glu");
  const long long total = static_cast<long long>(num_rows) * inter;
  if (total == 0) return 0;
  const unsigned blocks = static_cast<unsigned>((total + 255) / 256);
  if (dtype == 0)
    clamped_glu_kernel<__nv_bfloat16><<<blocks, 256, 0, as_stream(stream)>>>(
        static_cast<const __nv_bfloat16*>(gate_up), static_cast<__nv_bfloat16*>(out), total, inter, limit, alpha, shift);
  else
    clamped_glu_kernel<float><<<blocks, 256, 0, as_stream(stream)>>>(static_cast<const float*>(gate_up),
                                                                     static_cast<float*>(out), total, inter, limit, alpha, shift);
  B200_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int b200_argmax_rows(const float* logits, int64_t* out, int num_rows, int n, void* stream) {
  B200_REQUIRE(logits && out && num_rows >= 0 && n > 0, "argmax_rows: null pointer or empty rows");
  int rc = check_device(nullptr);
  if (rc) return rc;
  if (num_rows == 0) return 0;
  argmax_rows_kernel<<<num_rows, 256, 0, as_stream(stream)>>>(logits, reinterpret_cast<long long*>(out), n);
  B200_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int b200_gemm_f32(const float* x, const float* w, float* y, int num_rows, int groups, int out_features,
                             int in_features, int x_step, int w_step, int y_step, int x_cols, int y_cols, void* stream) {
  B200_REQUIRE(x && w && y, "gemm_f32: null pointer");
  B200_REQUIRE(num_rows >= 0 && groups > 0 && groups <= 65535 && out_features > 0 && in_features > 0 && in_features % 4 == 0 &&
                   x_step % 4 == 0 && x_cols % 4 == 0,
               "gemm_f32: rows %d, groups %d, N %d, K %d (K and x_step must be multiples of 4)", num_rows, groups,
               out_features, in_features);
  B200_REQUIRE((groups - 1) * x_step + in_features <= x_cols && (groups - 1) * y_step + out_features <= y_cols,
               "gemm_f32: the groups do not fit %d input and %d output columns", x_cols, y_cols);
  B200_REQUIRE(aligned16({x, w}), "gemm_f32: x and w must be 16-byte aligned");
  int rc = check_device(nullptr);
  if (rc) return rc;
  if (num_rows == 0) return 0;
  B200_REQUIRE((num_rows + 63) / 64 <= 65535, "gemm_f32: too many rows");
  const dim3 grid((out_features + 63) / 64, (num_rows + 63) / 64, groups);
  gemm_f32_kernel<<<grid, 256, 0, as_stream(stream)>>>(x, w, y, num_rows, out_features, in_features, x_step, w_step, y_step,
                                                       x_cols, y_cols, nullptr, nullptr, 0);
  B200_CUDA(cudaGetLastError());
  return 0;
}

extern "C" int b200_moe_gemm_f32(const float* x, const float* w, float* y, const void* tiles, const int32_t* num_tiles,
                                 int num_rows, int num_experts, int max_tiles, int out_features, int in_features, void* stream) {
  B200_REQUIRE(x && w && y && tiles && num_tiles, "moe_gemm_f32: null pointer");
  B200_REQUIRE(num_rows >= 0 && num_experts > 0 && max_tiles > 0 && max_tiles <= 65535 && out_features > 0 && in_features > 0 &&
                   in_features % 4 == 0,
               "moe_gemm_f32: %d rows, %d experts, at most %d tiles, N %d, K %d", num_rows, num_experts, max_tiles, out_features,
               in_features);
  B200_REQUIRE(aligned16({x, w}), "moe_gemm_f32: x and w must be 16-byte aligned");
  int rc = check_device(nullptr);
  if (rc) return rc;
  if (num_rows == 0) return 0;
  gemm_f32_kernel<<<dim3((out_features + 63) / 64, max_tiles), 256, 0, as_stream(stream)>>>(
      x, w, y, num_rows, out_features, in_features, 0, out_features, 0, in_features, out_features,
      static_cast<const MoeTile*>(tiles), num_tiles, num_experts);
  B200_CUDA(cudaGetLastError());
  return 0;
}
