// Attention whose scores are mixed over the query heads before the softmax, under a sliding window and with a penalty
// that grows with the distance (Sefalorn; engine: layered.py), over paged K/V.
//
//     own_g(i, j) = scale q_g . k_c(g),j - r1_g ln(1 + r2_g (i - j)),   score_h = sum_g T[h, g] own_g,   0 <= i - j < window
//
// Mixing is linear, so it is taken out of the score loop: score_h = Q'_h . K_j - B[h][i - j], where K_j are the keys of all kv
// heads side by side, Q'_h[c] = sum over the heads g of kv head c of T[h, g] scale q_g (mix_heads_kernel), and
// B[h][d] = sum_g T[h, g] r1_g ln(1 + r2_g d) is a table over the window's distances, kept in log2 units and padded with +inf on
// both sides (kDistPad, kDistTail): outside the window, and for later tokens, it masks.  Every query head then meets the whole
// of a token's keys, and the values of its own kv head.
//
// Pools are cut into 64-wide columns: [num_blocks, kv_heads * size / 64, page, 64], so that a page's keys (or values) of all heads
// are one run of 128-byte rows.
//
// Decode kernel: bf16.  grid (rows, splits); a CTA owns up to `split_tokens` consecutive
// tokens of one row, for all heads, and streams their pages (a producer warp, TMA boxes of up to 256 rows of 128 B, mbarrier ring
// of pages).  Groups of eight consumer warps take two pages (32 tokens) at a time:
//   scores   an item is (page, half of its tokens, 16 query heads): mma.sync m16n8k16 over the keys of all kv heads, queries
//            from shared memory; times log2 e, less the distance table, masked, into a score tile in shared memory
//   values   a unit is (kv head, 16 of its query heads, 64 value columns): online softmax over the tile's 32 tokens in the A
//            operand's registers, O += P V
// with one barrier of the group per two pages (the score tile is double-buffered).  Rows of one split are written as they are,
// others as fp32 partials that a second kernel folds in split order.
//
// Generic kernel: any sizes, bf16 or fp32, fp32 arithmetic, one CTA per (row, query head).

#include <type_traits>

#include "glue.cuh"

namespace b200 {

constexpr int kMixWarps = 4;
constexpr float kMixLog2e = 1.4426950408889634f;

struct MixedAttnParams {
  const void* q;            // [rows, heads, dk], or mixed already: [rows, heads, kv_heads * dk]
  const float* mix;         // [heads, heads]: q is raw and mix applies; NULL: q is mixed
  const void* k_pool;       // [num_blocks, kv_heads * dk / 64, page, 64]
  const void* v_pool;       // [num_blocks, kv_heads * dv / 64, page, 64]
  const int* table;         // [rows, max_pages], or one row for all (table_stride 0)
  int table_stride;
  const int* positions;     // [rows]: position of the row's token
  const float* bias;        // [heads, bias_ld], distance d at kDistPad + d
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
    const T* kr = kp + static_cast<size_t>(id) * K * p.page + slot * 64;
    for (int d = lane; d < K; d += 32) dot = fmaf(mg_sm[d], to_f32<T>(kr[(d >> 6) * p.page * 64 + (d & 63)]), dot);
    dot = fmaf(warp_sum(dot), kMixLog2e, -bias[kDistPad + pos - tok]);
    const float mn = fmaxf(m, dot);
    const float a = exp2f(m - mn), w = exp2f(dot - mn);
    m = mn;
    l = l * a + w;
    const T* vr = vp + (static_cast<size_t>(id) * p.kv_heads + kvh) * p.dv * p.page + slot * 64;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int d = lane + 32 * j;
      if (d < p.dv) acc[j] = acc[j] * a + w * to_f32<T>(vr[(d >> 6) * p.page * 64 + (d & 63)]);
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
      const float wgt = m_sm[w] == -INFINITY ? 0.f : exp2f(m_sm[w] - mmax);
      num += wgt * o_sm[w * p.dv + d];
      den += wgt * l_sm[w];
    }
    static_cast<T*>(p.out)[static_cast<size_t>(row) * p.out_ld + static_cast<size_t>(h) * p.dv + d] =
        from_f32<T>(den > 0.f ? p.out_scale * num / den : 0.f);
  }
}

constexpr int kMdPage = 16;
constexpr int kMdWarps = 8;                    // consumers of a group
constexpr int kMdScoreLd = 40;                 // floats per head of a score tile (32 tokens): float2 reads of 8 heads hit all banks
constexpr int kMdMergeFloats = 8 * 32 * 36;    // what the second group hands to the first

struct MixedDecodeParams {
  MixedAttnParams a;
  float* part_o;    // [rows, heads, max_splits, dv]
  float2* part_ml;
  int split_tokens, max_splits, stages;
  int k_box, v_box;  // rows of a TMA box: they divide a page's rows
};

// UNITS: units (see above) a warp may own.  GROUPS: groups of eight consumer warps; two of them take the tiles in turn, each with
// a softmax of its own, and are merged at the end.
template <int UNITS, int GROUPS>
__global__ void __launch_bounds__((GROUPS * kMdWarps + 1) * 32, 1)
mixed_decode_kernel(const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map, const MixedDecodeParams pp) {
#ifdef B200_DEVICE_OK
  const MixedAttnParams& p = pp.a;
  extern __shared__ uint8_t smem_raw[];
  grid_dep_wait();
  grid_dep_launch();
  const int row = blockIdx.x, split = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int pos = p.positions[row];
  if (pos < 0 || pos >= p.max_pages * kMdPage) {
    if (threadIdx.x == 0) set_error(p.err, kErrDevBadCtxLen);
    pos = 0;
  }
  const int lo = max(0, pos - p.window + 1);
  const int range0 = lo & ~(kMdPage - 1);
  const int start = range0 + split * pp.split_tokens;
  if (start > pos) return;  // uniform for the whole CTA
  const int nsplits = (pos + 1 - range0 + pp.split_tokens - 1) / pp.split_tokens;
  const int end = min(pos + 1, start + pp.split_tokens);
  const int npages = (end - start + kMdPage - 1) / kMdPage, first_page = start / kMdPage;

  const uint32_t ring = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* ring_ptr = smem_raw + (ring - smem_u32(smem_raw));
  const int kc = p.kv_heads * (p.dk / 64), vc = p.kv_heads * (p.dv / 64);  // 2 KiB boxes of a page
  const uint32_t stage_bytes = static_cast<uint32_t>(kc + vc) * 2048u;
  const int stages = pp.stages;
  uint8_t* after = ring_ptr + static_cast<size_t>(stages) * stage_bytes;
  const uint32_t bar_full = ring + stages * stage_bytes, bar_empty = bar_full + 8 * stages;  // up to 16 of each
  const int mt = (p.heads + 15) / 16, K = p.kv_heads * p.dk, q_ld = K + 8;
  const int score_floats = mt * 16 * kMdScoreLd;
  float* sc = reinterpret_cast<float*>(after + 256);     // [GROUPS][2][mt * 16][kMdScoreLd]
  __nv_bfloat16* q_sm = reinterpret_cast<__nv_bfloat16*>(sc + GROUPS * 2 * score_floats);  // [mt * 16][q_ld]

  if (threadIdx.x == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(bar_full + 8 * s, 1);
      mbar_init(bar_empty + 8 * s, kMdWarps);
    }
    fence_mbar_init();
    fence_proxy_async();
  }
  __syncthreads();

  if (warp == GROUPS * kMdWarps) {
    // ------------------------------------------------------------ producer --
    if (lane == 0) {
      tma_prefetch_desc(&k_map);
      tma_prefetch_desc(&v_map);
    }
    const int* table = p.table + static_cast<size_t>(row) * p.table_stride + first_page;
    const int k_boxes = (kc * kMdPage + pp.k_box - 1) / pp.k_box, v_boxes = (vc * kMdPage + pp.v_box - 1) / pp.v_box;
    int ids = 0, slot = 0;
    uint32_t phase = 1;
    for (int i = 0; i < npages; ++i) {
      if ((i & 31) == 0) {
        ids = i + lane < npages ? table[i + lane] : 0;
        if (ids < 0 || ids >= p.num_blocks) {
          set_error(p.err, kErrDevBadBlockId);
          ids = 0;
        }
      }
      const int id = __shfl_sync(0xffffffffu, ids, i & 31);
      if (!__all_sync(0xffffffffu, mbar_wait(bar_empty + 8 * slot, phase, p.err))) break;
      if (lane == 0) mbar_arrive_expect_tx(bar_full + 8 * slot, stage_bytes);
      __syncwarp();
      for (int b = lane; b < k_boxes + v_boxes; b += 32) {
        if (b < k_boxes)
          tma_load_2d(ring + slot * stage_bytes + b * pp.k_box * 128u, &k_map, bar_full + 8 * slot, 0, id * kc * kMdPage + b * pp.k_box);
        else
          tma_load_2d(ring + slot * stage_bytes + kc * 2048u + (b - k_boxes) * pp.v_box * 128u, &v_map, bar_full + 8 * slot, 0,
                      id * vc * kMdPage + (b - k_boxes) * pp.v_box);
      }
      if (++slot == stages) {
        slot = 0;
        phase ^= 1;
      }
    }
    if (GROUPS > 1) asm volatile("bar.sync 3, %0;" ::"n"((GROUPS * kMdWarps + 1) * 32) : "memory");
    return;
  }

  // ------------------------------------------------------------- consumers --
  const int group = GROUPS > 1 ? warp / kMdWarps : 0, w = warp - group * kMdWarps;
  const int per = p.heads / p.kv_heads;
  if (p.mix == nullptr) {  // the row's mixed queries, zero rows after the last head
    const uint4* src = reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.q) + static_cast<size_t>(row) * p.heads * K);
    const int per_row = K / 8;
    for (int i = threadIdx.x; i < mt * 16 * per_row; i += GROUPS * kMdWarps * 32) {
      const int h = i / per_row, c = i - h * per_row;
      *reinterpret_cast<uint4*>(q_sm + static_cast<size_t>(h) * q_ld + c * 8) = h < p.heads ? src[i] : make_uint4(0u, 0u, 0u, 0u);
    }
  } else {  // mix them here: an item is eight columns of one kv head's key and a range of heads (at most 8 raw queries)
    const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(p.q) + static_cast<size_t>(row) * p.heads * p.dk;
    const int d8 = p.dk / 8, cols = p.kv_heads * d8;
    const int ranges = max(1, GROUPS * kMdWarps * 32 / cols), span = (mt * 16 + ranges - 1) / ranges;
    for (int i = threadIdx.x; i < cols * ranges; i += GROUPS * kMdWarps * 32) {
      const int rg = i / cols, cd = i - rg * cols, c = cd / d8, d = (cd - c * d8) * 8;
      const int h_end = min(mt * 16, (rg + 1) * span);
      float q8[8][8];
#pragma unroll
      for (int g = 0; g < 8; ++g) {
        if (g < per) {
          load8<__nv_bfloat16>(src + (c * per + g) * p.dk + d, q8[g]);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) q8[g][e] = 0.f;
        }
      }
      for (int h = rg * span; h < h_end; ++h) {
        float acc[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[e] = 0.f;
        if (h < p.heads) {
          const float* m = p.mix + static_cast<size_t>(h) * p.heads + c * per;
#pragma unroll
          for (int g = 0; g < 8; ++g) {
            if (g >= per) break;
            const float mv = __ldg(m + g);
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[e] = fmaf(mv, q8[g][e], acc[e]);
          }
        }
        store8<__nv_bfloat16>(q_sm + static_cast<size_t>(h) * q_ld + c * p.dk + d, acc);
      }
    }
  }
  const int sub = (per + 15) / 16, dvc = p.dv / 64;
  const int units = p.kv_heads * sub * dvc;
  const int gq = lane >> 2, tq = lane & 3;
  const int lj = lane >> 3, lr = lane & 7;
  float o[UNITS][8][4], m_run[UNITS][2], l_run[UNITS][2];
  int s_off[UNITS][2], v_off[UNITS];  // score rows and value boxes of this warp's units; v_off < 0: no such unit
#pragma unroll
  for (int u = 0; u < UNITS; ++u) {
#pragma unroll
    for (int n = 0; n < 8; ++n) o[u][n][0] = o[u][n][1] = o[u][n][2] = o[u][n][3] = 0.f;
    m_run[u][0] = m_run[u][1] = -INFINITY;
    l_run[u][0] = l_run[u][1] = 0.f;
    const int unit = w + u * kMdWarps, hs = unit / dvc, c = hs / sub, h0 = (hs - c * sub) * 16 + gq;
    const bool is = unit < units;
    s_off[u][0] = is ? (c * per + min(h0, per - 1)) * kMdScoreLd + 2 * tq : 0;  // a row past the last head repeats it and is not kept
    s_off[u][1] = is ? (c * per + min(h0 + 8, per - 1)) * kMdScoreLd + 2 * tq : 0;
    v_off[u] = is ? (kc + c * dvc + (unit - hs * dvc)) * 2048 : -1;
  }
  const uint32_t v_sw = swz128((lj & 1) * 8 + lr, lj >> 1);  // value columns 16 further: ^ 32, ^ 64, ^ 96
  // All 16 warps: queries in place.
  if (GROUPS > 1) asm volatile("bar.sync 4, %0;" ::"n"(GROUPS * kMdWarps * 32) : "memory");
  else asm volatile("bar.sync 4, %0;" ::"n"(kMdWarps * 32) : "memory");
  const uint32_t a_base = smem_u32(q_sm) + (((lj & 1) * 8 + lr) * q_ld + (lj >> 1) * 8) * 2;

  bool alive = true;
  const int tiles = (npages + 1) / 2;
  // this group's first page in the ring, and its parity
  int slot = group * 2;
  uint32_t phase = 0;
  while (slot >= stages) {
    slot -= stages;
    phase ^= 1;
  }
#pragma unroll 1
  for (int tile = group, turn = 0; tile < tiles; tile += GROUPS, ++turn) {
    const int pages_here = min(2, npages - tile * 2);
    int slot1 = slot + 1;
    uint32_t phase1 = phase;
    if (slot1 == stages) {
      slot1 = 0;
      phase1 ^= 1;
    }
    float* score = sc + (group * 2 + (turn & 1)) * score_floats;
    const int tok_tile = start + tile * 2 * kMdPage;
    if (alive) alive = mbar_wait(bar_full + 8 * slot, phase, p.err);
    if (pages_here > 1 && alive) alive = mbar_wait(bar_full + 8 * slot1, phase1, p.err);
    // ---- scores: an item is 16 heads and a page, or half a page where there are too few heads to keep all warps busy so
    const auto score_item = [&](auto halves, int pg, int th0, int mi) {
      constexpr int NT = decltype(halves)::value;
      // the distance table's entries travel while the products run
      const float* bt = p.bias + static_cast<size_t>(mi * 16 + gq) * p.bias_ld + (kDistPad + pos - tok_tile - pg * 16 - th0 * 8 - 2 * tq);
      const bool h_lo = mi * 16 + gq < p.heads, h_hi = mi * 16 + gq + 8 < p.heads;
      const size_t b_hi = static_cast<size_t>(8) * p.bias_ld;
      float b[NT][4], acc[NT][2][4];
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        b[t][0] = h_lo ? __ldg(bt - t * 8) : 0.f;
        b[t][1] = h_lo ? __ldg(bt - t * 8 - 1) : 0.f;
        b[t][2] = h_hi ? __ldg(bt - t * 8 + b_hi) : 0.f;
        b[t][3] = h_hi ? __ldg(bt - t * 8 + b_hi - 1) : 0.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[t][0][e] = acc[t][1][e] = 0.f;
      }
      uint32_t a_addr = a_base + mi * 16 * q_ld * 2;
      uint32_t k_lo = ring + (pg ? slot1 : slot) * stage_bytes + swz128(th0 * 8 + lr, lj);  // 8 tokens further: + 1 KiB
#pragma unroll 4
      for (int c = 0; c < kc; ++c) {  // 64 of the key columns
        uint32_t a0[4], a1[4], a2[4], a3[4];
        ldmatrix_x4(a_addr, a0[0], a0[1], a0[2], a0[3]);
        ldmatrix_x4(a_addr + 32, a1[0], a1[1], a1[2], a1[3]);
        ldmatrix_x4(a_addr + 64, a2[0], a2[1], a2[2], a2[3]);
        ldmatrix_x4(a_addr + 96, a3[0], a3[1], a3[2], a3[3]);
#pragma unroll
        for (int t = 0; t < NT; ++t) {
          uint32_t b0, b1, b2, b3, b4, b5, b6, b7;
          ldmatrix_x4(k_lo + t * 1024, b0, b1, b2, b3);
          ldmatrix_x4((k_lo ^ 64u) + t * 1024, b4, b5, b6, b7);
          mma_bf16_16816(acc[t][0], a0, b0, b1);
          mma_bf16_16816(acc[t][1], a1, b2, b3);
          mma_bf16_16816(acc[t][0], a2, b4, b5);
          mma_bf16_16816(acc[t][1], a3, b6, b7);
        }
        k_lo += 2048u;
        a_addr += 128u;
      }
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        const float *x = acc[t][0], *y = acc[t][1];
        float* dst = score + (mi * 16 + gq) * kMdScoreLd + pg * 16 + (th0 + t) * 8 + 2 * tq;
        *reinterpret_cast<float2*>(dst) = make_float2(fmaf(x[0] + y[0], kMixLog2e, -b[t][0]), fmaf(x[1] + y[1], kMixLog2e, -b[t][1]));
        *reinterpret_cast<float2*>(dst + 8 * kMdScoreLd) =
            make_float2(fmaf(x[2] + y[2], kMixLog2e, -b[t][2]), fmaf(x[3] + y[3], kMixLog2e, -b[t][3]));
      }
    };
    constexpr bool kWide = UNITS <= 2 && GROUPS == 1;  // elsewhere the registers are needed
    if (kWide && mt * 2 >= kMdWarps) {
#pragma unroll 1
      for (int item = w; item < mt * 2; item += kMdWarps)
        if ((item & 1) < pages_here) score_item(std::integral_constant<int, kWide ? 2 : 1>{}, item & 1, 0, item >> 1);
    } else {
#pragma unroll 1
      for (int item = w; item < mt * 4; item += kMdWarps)
        if ((item & 1) < pages_here) score_item(std::integral_constant<int, 1>{}, item & 1, (item >> 1) & 1, item >> 2);
    }
    // the group's score tile is complete, and its other one has been read by all its warps
    asm volatile("bar.sync %0, %1;" ::"r"(1 + group), "n"(kMdWarps * 32) : "memory");
    // ---- values
#pragma unroll
    for (int u = 0; u < UNITS; ++u) {
      if (v_off[u] < 0) break;
      const float* s0 = score + s_off[u][0];
      const float* s1 = score + s_off[u][1];
      float s[2][2][4];  // [page][row half][k 2tq, 2tq+1, 2tq+8, 2tq+9]
#pragma unroll
      for (int pg = 0; pg < 2; ++pg) {
        if (pg == 0 || pages_here > 1) {
          const float2 a = *reinterpret_cast<const float2*>(s0 + pg * 16), b = *reinterpret_cast<const float2*>(s0 + pg * 16 + 8);
          const float2 x = *reinterpret_cast<const float2*>(s1 + pg * 16), y = *reinterpret_cast<const float2*>(s1 + pg * 16 + 8);
          s[pg][0][0] = a.x; s[pg][0][1] = a.y; s[pg][0][2] = b.x; s[pg][0][3] = b.y;
          s[pg][1][0] = x.x; s[pg][1][1] = x.y; s[pg][1][2] = y.x; s[pg][1][3] = y.y;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) s[pg][0][e] = s[pg][1][e] = -INFINITY;
        }
      }
      float mx0 = s[0][0][0], mx1 = s[0][1][0];
#pragma unroll
      for (int e = 1; e < 8; ++e) {
        mx0 = fmaxf(mx0, s[e >> 2][0][e & 3]);
        mx1 = fmaxf(mx1, s[e >> 2][1][e & 3]);
      }
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
      const float n0 = fmaxf(m_run[u][0], mx0), n1 = fmaxf(m_run[u][1], mx1);
      const float r0 = n0 == -INFINITY ? 0.f : n0, r1 = n1 == -INFINITY ? 0.f : n1;  // nothing seen yet: all weights come out 0
      if (__any_sync(0xffffffffu, n0 != m_run[u][0] || n1 != m_run[u][1])) {
        const float al0 = fast_ex2(m_run[u][0] - r0), al1 = fast_ex2(m_run[u][1] - r1);
        m_run[u][0] = n0;
        m_run[u][1] = n1;
        l_run[u][0] *= al0;
        l_run[u][1] *= al1;
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          o[u][n][0] *= al0;
          o[u][n][1] *= al0;
          o[u][n][2] *= al1;
          o[u][n][3] *= al1;
        }
      }
      uint32_t pa[2][4];
#pragma unroll
      for (int pg = 0; pg < 2; ++pg) {
        float e0[4], e1[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          e0[e] = fast_ex2(s[pg][0][e] - r0);
          e1[e] = fast_ex2(s[pg][1][e] - r1);
        }
        l_run[u][0] += (e0[0] + e0[1]) + (e0[2] + e0[3]);
        l_run[u][1] += (e1[0] + e1[1]) + (e1[2] + e1[3]);
        pa[pg][0] = pack_bf16x2(e0[0], e0[1]);
        pa[pg][1] = pack_bf16x2(e1[0], e1[1]);
        pa[pg][2] = pack_bf16x2(e0[2], e0[3]);
        pa[pg][3] = pack_bf16x2(e1[2], e1[3]);
      }
#pragma unroll
      for (int pg = 0; pg < 2; ++pg) {
        if (pg > 0 && pages_here < 2) break;
        const uint32_t vbase = ring + (pg ? slot1 : slot) * stage_bytes + v_off[u] + v_sw;
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          uint32_t v0, v1, v2, v3;
          ldmatrix_x4_trans(vbase ^ (np * 32u), v0, v1, v2, v3);
          mma_bf16_16816(o[u][2 * np], pa[pg], v0, v1);
          mma_bf16_16816(o[u][2 * np + 1], pa[pg], v2, v3);
        }
      }
    }
    __syncwarp();
    if (lane == 0) {
      mbar_arrive(bar_empty + 8 * slot);
      if (pages_here > 1) mbar_arrive(bar_empty + 8 * slot1);
    }
    slot += 2 * GROUPS;
    while (slot >= stages) {
      slot -= stages;
      phase ^= 1;
    }
  }

#pragma unroll
  for (int u = 0; u < UNITS; ++u)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      l_run[u][hh] += __shfl_xor_sync(0xffffffffu, l_run[u][hh], 1);
      l_run[u][hh] += __shfl_xor_sync(0xffffffffu, l_run[u][hh], 2);
    }
  if (GROUPS > 1) {  // every page has been read: the second group's results go through the ring
    float* mg = reinterpret_cast<float*>(ring_ptr) + (w * 36) * 32 + lane;
    // all copies have landed and been read (the producer has issued its last one before it comes here)
    asm volatile("bar.sync 3, %0;" ::"n"((GROUPS * kMdWarps + 1) * 32) : "memory");
    if (group == 1) {
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) mg[(n * 4 + e) * 32] = o[0][n][e];
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        mg[(32 + hh) * 32] = m_run[0][hh];
        mg[(34 + hh) * 32] = l_run[0][hh];
      }
    }
    asm volatile("bar.sync 4, %0;" ::"n"(GROUPS * kMdWarps * 32) : "memory");
    if (group == 1) return;
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const float m1 = mg[(32 + hh) * 32], l1 = mg[(34 + hh) * 32], m0 = m_run[0][hh];
      const float m = fmaxf(m0, m1), r = m == -INFINITY ? 0.f : m;
      const float c0 = fast_ex2(m0 - r), c1 = fast_ex2(m1 - r);
      m_run[0][hh] = m;
      l_run[0][hh] = l_run[0][hh] * c0 + l1 * c1;
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 2 * hh; e < 2 * hh + 2; ++e) o[0][n][e] = o[0][n][e] * c0 + mg[(n * 4 + e) * 32] * c1;
    }
  }

#pragma unroll
  for (int u = 0; u < UNITS; ++u) {
    const int unit = w + u * kMdWarps;
    if (unit >= units) break;
    const int vcol = unit % dvc, hs = unit / dvc, c = hs / sub, ms = hs - c * sub;
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int hl = ms * 16 + gq + hh * 8;
      if (hl >= per) continue;
      const int h = c * per + hl;
      if (nsplits == 1) {
        const float inv = p.out_scale / l_run[u][hh];
        __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + static_cast<size_t>(row) * p.out_ld + static_cast<size_t>(h) * p.dv + vcol * 64;
#pragma unroll
        for (int n = 0; n < 8; ++n)
          *reinterpret_cast<uint32_t*>(dst + n * 8 + 2 * tq) = pack_bf16x2(o[u][n][2 * hh] * inv, o[u][n][2 * hh + 1] * inv);
      } else {
        const size_t at = (static_cast<size_t>(row) * p.heads + h) * pp.max_splits + split;
#pragma unroll
        for (int n = 0; n < 8; ++n)
          *reinterpret_cast<float2*>(pp.part_o + at * p.dv + vcol * 64 + n * 8 + 2 * tq) = make_float2(o[u][n][2 * hh], o[u][n][2 * hh + 1]);
        if (vcol == 0 && tq == 0) pp.part_ml[at] = make_float2(m_run[u][hh], l_run[u][hh]);
      }
    }
  }
#endif
}

// Folds the partials of one (row, head) in split order; rows of one split are already written.  A warp per (row, head).
__global__ void __launch_bounds__(128)
mixed_reduce_kernel(const MixedDecodeParams pp) {
  const MixedAttnParams& p = pp.a;
  grid_dep_wait();
  grid_dep_launch();
  const int item = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= p.rows * p.heads) return;
  const int row = item / p.heads, h = item - row * p.heads;
  int pos = p.positions[row];
  if (pos < 0 || pos >= p.max_pages * kMdPage) pos = 0;
  const int range0 = max(0, pos - p.window + 1) & ~(kMdPage - 1);
  const int n = (pos + 1 - range0 + pp.split_tokens - 1) / pp.split_tokens;
  if (n <= 1) return;
  const size_t base = static_cast<size_t>(item) * pp.max_splits;
  float m = -INFINITY;
  for (int s = lane; s < n; s += 32) m = fmaxf(m, pp.part_ml[base + s].x);
  m = warp_max(m);
  float den = 0.f;
  for (int s = lane; s < n; s += 32) {
    const float2 ml = pp.part_ml[base + s];
    den += exp2f(ml.x - m) * ml.y;
  }
  const float inv = p.out_scale / warp_sum(den);
  __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + static_cast<size_t>(row) * p.out_ld + static_cast<size_t>(h) * p.dv;
  for (int d = lane * 2; d < p.dv; d += 64) {
    float a = 0.f, b = 0.f;
#pragma unroll 4
    for (int s = 0; s < n; ++s) {
      const float w = exp2f(pp.part_ml[base + s].x - m);
      const float2 v = *reinterpret_cast<const float2*>(pp.part_o + (base + s) * p.dv + d);
      a = fmaf(w, v.x, a);
      b = fmaf(w, v.y, b);
    }
    *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16x2(a * inv, b * inv);
  }
}

// Splits of the longest window.
static int mixed_max_splits(int window, int max_pages, int split_tokens) {
  const long long all = static_cast<long long>(max_pages) * kMdPage;
  long long seen = (static_cast<long long>(window) + kMdPage - 1) / kMdPage * kMdPage + kMdPage;
  if (seen > all) seen = all;
  return static_cast<int>((seen + split_tokens - 1) / split_tokens);
}

// Pages in flight, groups of consumer warps and shared memory of the decode kernel; 0: not built for this shape.
static int mixed_decode_stages(int heads, int kv_heads, int dk, int dv, size_t* smem_out, int* groups_out) {
  if (heads % kv_heads || dk % 64 || dv % 64) return 0;
  const int per = heads / kv_heads, units = kv_heads * ((per + 15) / 16) * (dv / 64);
  if (units > 4 * kMdWarps) return 0;
  const size_t mt = (heads + 15) / 16, K = static_cast<size_t>(kv_heads) * dk;
  const size_t stage = static_cast<size_t>(kv_heads) * (dk + dv) / 64 * 2048, room = 227 * 1024;
  const auto fixed = [&](int groups) { return 1024 + 256 + groups * 2 * mt * 16 * kMdScoreLd * 4 + mt * 16 * (K + 8) * 2; };
  // two groups where their accumulators fit the registers and five pages the shared memory
  int groups = units <= kMdWarps && fixed(2) + 5 * stage <= room && 5 * stage >= kMdMergeFloats * 4 ? 2 : 1;
  if (fixed(groups) + 3 * stage > room) return 0;
  size_t stages = (room - fixed(groups)) / stage;
  if (stages > 16) stages = 16;
  if (smem_out) *smem_out = fixed(groups) + stages * stage;
  if (groups_out) *groups_out = groups;
  return static_cast<int>(stages);
}

template <int UNITS, int GROUPS>
static int launch_mixed_decode(const CUtensorMap& km, const CUtensorMap& vm, const MixedDecodeParams& pp, size_t smem, cudaStream_t st) {
  int rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&mixed_decode_kernel<UNITS, GROUPS>), 227 * 1024);
  if (rc) return rc;
  B200_CUDA(launch_overlapped(mixed_decode_kernel<UNITS, GROUPS>, dim3(pp.a.rows, pp.max_splits), dim3((GROUPS * kMdWarps + 1) * 32), smem, st, km, vm, pp));
  if (pp.max_splits > 1)
    B200_CUDA(launch_overlapped(mixed_reduce_kernel, dim3((pp.a.rows * pp.a.heads + 3) / 4), dim3(128), 0, st, pp));
  return 0;
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

extern "C" size_t b200_mixed_attn_workspace_bytes(int num_rows, int num_q_heads, int num_kv_heads, int key_dim, int value_dim,
                                                  int window, int max_pages_per_seq, int split_tokens) {
  if (num_rows <= 0 || num_q_heads <= 0 || num_kv_heads <= 0 || key_dim <= 0 || value_dim <= 0 || window <= 0 ||
      max_pages_per_seq <= 0 || split_tokens <= 0 || mixed_decode_stages(num_q_heads, num_kv_heads, key_dim, value_dim, nullptr, nullptr) == 0)
    return 256;
  return carve(nullptr, num_rows, num_q_heads, value_dim, mixed_max_splits(window, max_pages_per_seq, split_tokens)).bytes;
}

extern "C" int b200_mixed_attn_mixes(int num_q_heads, int num_kv_heads, int key_dim, int value_dim) {
  // a kv head's raw queries sit in registers
  return num_kv_heads > 0 && num_q_heads % num_kv_heads == 0 && num_q_heads / num_kv_heads <= 8 &&
         mixed_decode_stages(num_q_heads, num_kv_heads, key_dim, value_dim, nullptr, nullptr) > 0;
}

extern "C" int b200_mixed_attn(const void* q, const float* mix, const void* k_pool, const void* v_pool, const int32_t* block_table,
                               int table_stride, const int32_t* positions, const float* bias, int bias_ld, int window,
                               void* out, int out_ld, float out_scale, void* workspace, size_t workspace_bytes,
                               void* status_word, int num_rows, int num_q_heads, int num_kv_heads, int key_dim, int value_dim,
                               int page_size, int num_blocks, int max_pages_per_seq, int split_tokens, int dtype, void* stream) {
  B200_REQUIRE(q && k_pool && v_pool && block_table && positions && bias && out, "mixed_attn: null pointer");
  B200_REQUIRE(num_rows >= 0 && num_rows <= 65535 && num_q_heads > 0 && num_kv_heads > 0 && num_q_heads % num_kv_heads == 0 &&
                   key_dim > 0 && value_dim > 0 && key_dim % 64 == 0 && value_dim % 64 == 0 && value_dim <= 1024 && page_size > 0 && num_blocks > 0 &&
                   max_pages_per_seq > 0 && window > 0 && (table_stride == 0 || table_stride >= max_pages_per_seq),
               "mixed_attn: %d rows, %d query heads over %d, key size %d, value size %d, window %d", num_rows, num_q_heads,
               num_kv_heads, key_dim, value_dim, window);
  const long long all = static_cast<long long>(max_pages_per_seq) * page_size;
  B200_REQUIRE(bias_ld >= kDistPad + (window < all ? window : all) + kDistTail && out_ld >= num_q_heads * value_dim,
               "mixed_attn: bias rows of %d for a window of %d, output rows of %d", bias_ld, window, out_ld);
  B200_GLUE_DTYPE("mixed_attn");
  if (num_rows == 0) return 0;
  const MixedAttnParams p{q, mix, k_pool, v_pool, block_table, table_stride, positions, bias, bias_ld, window, out, out_ld,
                          out_scale, static_cast<int*>(status_word), num_rows, num_q_heads, num_kv_heads, key_dim, value_dim,
                          page_size, num_blocks, max_pages_per_seq};
  B200_REQUIRE(mix == nullptr || (dtype == 0 && page_size == kMdPage && split_tokens > 0 &&
                                  b200_mixed_attn_mixes(num_q_heads, num_kv_heads, key_dim, value_dim)),
               "mixed_attn: raw queries of %d heads over %d cannot be mixed here", num_q_heads, num_kv_heads);
  size_t smem = 0;
  int groups = 1;
  const int stages = dtype == 0 && page_size == kMdPage && split_tokens > 0
                         ? mixed_decode_stages(num_q_heads, num_kv_heads, key_dim, value_dim, &smem, &groups) : 0;
  if (stages > 0) {
    B200_REQUIRE(split_tokens % 32 == 0 && out_ld % 2 == 0, "mixed_attn: split_tokens %d is no multiple of 32", split_tokens);
    B200_REQUIRE(aligned16({q, k_pool, v_pool}) && (reinterpret_cast<uintptr_t>(out) & 3) == 0, "mixed_attn: buffers must be aligned");
    MixedDecodeParams pp{p, nullptr, nullptr, split_tokens, mixed_max_splits(window, max_pages_per_seq, split_tokens), stages, 0, 0};
    B200_REQUIRE(pp.max_splits <= 65535, "mixed_attn: grid too large");
    if (pp.max_splits > 1) {
      const AttnWorkspace w = carve(workspace, num_rows, num_q_heads, value_dim, pp.max_splits);
      if (workspace == nullptr || workspace_bytes < w.bytes) {
        set_detail("mixed_attn: workspace %zu < required %zu", workspace_bytes, w.bytes);
        return -kErrWorkspace;
      }
      pp.part_o = w.o;
      pp.part_ml = w.ml;
    }
    CUtensorMap km, vm;
    const auto box_rows = [](int rows) {  // of 128 bytes, a page's: the largest equal parts of at most 256
      int parts = (rows + 255) / 256;
      while (rows % parts) ++parts;
      return rows / parts;
    };
    const int k_rows = num_kv_heads * key_dim / 64 * kMdPage, v_rows = num_kv_heads * value_dim / 64 * kMdPage;
    pp.k_box = box_rows(k_rows);
    pp.v_box = box_rows(v_rows);
    int rc = get_tensor_map_2d(k_pool, static_cast<uint64_t>(num_blocks) * k_rows, 64, 2, pp.k_box, 64, &km);
    if (rc) return rc;
    rc = get_tensor_map_2d(v_pool, static_cast<uint64_t>(num_blocks) * v_rows, 64, 2, pp.v_box, 64, &vm);
    if (rc) return rc;
    const int per = num_q_heads / num_kv_heads, units = num_kv_heads * ((per + 15) / 16) * (value_dim / 64);
    if (groups == 2) return launch_mixed_decode<1, 2>(km, vm, pp, smem, as_stream(stream));
    if (units <= kMdWarps) return launch_mixed_decode<1, 1>(km, vm, pp, smem, as_stream(stream));
    if (units <= 2 * kMdWarps) return launch_mixed_decode<2, 1>(km, vm, pp, smem, as_stream(stream));
    return launch_mixed_decode<4, 1>(km, vm, pp, smem, as_stream(stream));
  }
  return dtype == 0 ? launch_mixed_generic<__nv_bfloat16>(p, as_stream(stream)) : launch_mixed_generic<float>(p, as_stream(stream));
}
