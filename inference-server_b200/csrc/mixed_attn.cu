// Attention whose scores are mixed over the query heads before the softmax, under a sliding window and with a penalty
// that grows with the distance (Sefalorn; engine: layered.py), over paged K/V.
//
//     own_g(i, j) = scale q_g . k_c(g),j - r1_g ln(1 + r2_g (i - j)),   score_h = sum_g T[h, g] own_g,   0 <= i - j < window
//
// Mixing is linear, so it is taken out of the score loop: score_h = Q'_h . K_j - B[h][i - j], where K_j are the keys of all kv
// heads side by side, Q'_h[c] = sum over the heads g of kv head c of T[h, g] scale q_g (mix_heads_kernel), and
// B[h][d] = sum_g T[h, g] r1_g ln(1 + r2_g d) is a table over the window's distances.  Every query head then meets the whole
// of a token's keys, and the values of its own kv head.
//
// Generic kernel (here): any sizes, bf16 or fp32, fp32 arithmetic, one CTA per (row, query head).

#include "glue.cuh"

namespace b200 {

constexpr int kMixWarps = 4;

struct MixedAttnParams {
  const void* q;            // [rows, heads, kv_heads * dk]
  const void* k_pool;       // [num_blocks, kv_heads, page, dk]
  const void* v_pool;       // [num_blocks, kv_heads, page, dv]
  const int* table;         // [rows, max_pages], or one row for all (table_stride 0)
  int table_stride;
  const int* positions;     // [rows]: position of the row's token
  const float* bias;        // [heads, bias_ld]
  int bias_ld, window;
  void* out;                // [rows, out_ld], head h at column h * dv
  int out_ld;
  float out_scale;
  int* err;
  int rows, heads, kv_heads, dk, dv, page, num_blocks, max_pages;
};

// PER: value columns per lane.
template <typename T, int PER>
__global__ void __launch_bounds__(kMixWarps * 32)
mixed_attn_generic_kernel(const MixedAttnParams p) {
  extern __shared__ float mg_sm[];  // q [kv_heads * dk], then o [warps, dv]
  __shared__ float m_sm[kMixWarps], l_sm[kMixWarps];
  grid_dep_wait();
  grid_dep_launch();
  const int h = blockIdx.x, row = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvh = h / (p.heads / p.kv_heads), K = p.kv_heads * p.dk;
  const T* q = static_cast<const T*>(p.q) + (static_cast<size_t>(row) * p.heads + h) * K;
  for (int i = threadIdx.x; i < K; i += blockDim.x) mg_sm[i] = to_f32<T>(q[i]);
  __syncthreads();
  const PageMap pm{p.page, p.num_blocks, p.max_pages, p.err};
  const int* table = p.table + static_cast<size_t>(row) * p.table_stride;
  int pos = p.positions[row];
  if (pos < 0 || pos >= p.max_pages * p.page) {
    if (threadIdx.x == 0) set_error(p.err, kErrDevBadCtxLen);
    pos = 0;
  }
  const T* kp = static_cast<const T*>(p.k_pool);
  const T* vp = static_cast<const T*>(p.v_pool);
  const float* bias = p.bias + static_cast<size_t>(h) * p.bias_ld;
  float acc[PER];
#pragma unroll
  for (int j = 0; j < PER; ++j) acc[j] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int tok = max(0, pos - p.window + 1) + warp; tok <= pos; tok += kMixWarps) {
    const int id = page_of(pm, table, tok);
    if (id < 0) continue;
    const int slot = tok % p.page;
    float dot = 0.f;
    for (int c = 0; c < p.kv_heads; ++c) {
      const T* kr = kp + ((static_cast<size_t>(id) * p.kv_heads + c) * p.page + slot) * p.dk;
      for (int d = lane; d < p.dk; d += 32) dot = fmaf(mg_sm[c * p.dk + d], to_f32<T>(kr[d]), dot);
    }
    dot = warp_sum(dot) - bias[min(pos - tok, p.bias_ld - 1)];
    const float mn = fmaxf(m, dot);
    const float a = expf(m - mn), w = expf(dot - mn);
    m = mn;
    l = l * a + w;
    const T* vr = vp + ((static_cast<size_t>(id) * p.kv_heads + kvh) * p.page + slot) * p.dv;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int d = lane + 32 * j;
      if (d < p.dv) acc[j] = acc[j] * a + w * to_f32<T>(vr[d]);
    }
  }
  float* o_sm = mg_sm + K;
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int d = lane + 32 * j;
    if (d < p.dv) o_sm[warp * p.dv + d] = acc[j];
  }
  if (lane == 0) {
    m_sm[warp] = m;
    l_sm[warp] = l;
  }
  __syncthreads();
  float mmax = -INFINITY;
  for (int w = 0; w < kMixWarps; ++w) mmax = fmaxf(mmax, m_sm[w]);
  for (int d = threadIdx.x; d < p.dv; d += blockDim.x) {
    float num = 0.f, den = 0.f;
    for (int w = 0; w < kMixWarps; ++w) {
      const float wgt = m_sm[w] == -INFINITY ? 0.f : expf(m_sm[w] - mmax);
      num += wgt * o_sm[w * p.dv + d];
      den += wgt * l_sm[w];
    }
    static_cast<T*>(p.out)[static_cast<size_t>(row) * p.out_ld + static_cast<size_t>(h) * p.dv + d] =
        from_f32<T>(den > 0.f ? p.out_scale * num / den : 0.f);
  }
}

template <typename T>
static int launch_mixed_generic(const MixedAttnParams& p, cudaStream_t st) {
  const size_t smem = (static_cast<size_t>(p.kv_heads) * p.dk + static_cast<size_t>(kMixWarps) * p.dv) * 4;
  B200_REQUIRE(smem <= 200 * 1024, "mixed_attn: %d kv heads of %d do not fit", p.kv_heads, p.dk);
#define B200_MIXED(PER)                                                                                               \
  do {                                                                                                                \
    int rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&mixed_attn_generic_kernel<T, PER>), 200 * 1024);      \
    if (rc) return rc;                                                                                                \
    B200_CUDA(launch_overlapped(mixed_attn_generic_kernel<T, PER>, dim3(p.heads, p.rows), dim3(kMixWarps * 32), smem, st, p)); \
  } while (0)
  if (p.dv <= 256) B200_MIXED(8);
  else B200_MIXED(32);
#undef B200_MIXED
  return 0;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_mixed_attn(const void* q, const void* k_pool, const void* v_pool, const int32_t* block_table,
                               int table_stride, const int32_t* positions, const float* bias, int bias_ld, int window,
                               void* out, int out_ld, float out_scale, void* status_word, int num_rows, int num_q_heads,
                               int num_kv_heads, int key_dim, int value_dim, int page_size, int num_blocks,
                               int max_pages_per_seq, int dtype, void* stream) {
  B200_REQUIRE(q && k_pool && v_pool && block_table && positions && bias && out, "mixed_attn: null pointer");
  B200_REQUIRE(num_rows >= 0 && num_rows <= 65535 && num_q_heads > 0 && num_kv_heads > 0 && num_q_heads % num_kv_heads == 0 &&
                   key_dim > 0 && value_dim > 0 && value_dim <= 1024 && page_size > 0 && num_blocks > 0 &&
                   max_pages_per_seq > 0 && window > 0 && (table_stride == 0 || table_stride >= max_pages_per_seq),
               "mixed_attn: %d rows, %d query heads over %d, key size %d, value size %d, window %d", num_rows, num_q_heads,
               num_kv_heads, key_dim, value_dim, window);
  const long long all = static_cast<long long>(max_pages_per_seq) * page_size;
  B200_REQUIRE(bias_ld >= (window < all ? window : all) && out_ld >= num_q_heads * value_dim,
               "mixed_attn: bias rows of %d for a window of %d, output rows of %d", bias_ld, window, out_ld);
  B200_GLUE_DTYPE("mixed_attn");
  if (num_rows == 0) return 0;
  const MixedAttnParams p{q, k_pool, v_pool, block_table, table_stride, positions, bias, bias_ld, window, out, out_ld,
                          out_scale, static_cast<int*>(status_word), num_rows, num_q_heads, num_kv_heads, key_dim, value_dim,
                          page_size, num_blocks, max_pages_per_seq};
  return dtype == 0 ? launch_mixed_generic<__nv_bfloat16>(p, as_stream(stream)) : launch_mixed_generic<float>(p, as_stream(stream));
}
