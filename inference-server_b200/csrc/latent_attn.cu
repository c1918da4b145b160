// Decode attention over a cache of latents for sm_100a.
//
// In latent attention a token leaves ONE vector c of `rank` numbers in the cache, and the keys and values of every head
// are linear maps of it: k_h = U_h c, v_h = V_h c.  A decode step does not form them: q_h . (U_h c) = (U_h^T q_h) . c,
// so the projected query q'_h = U_h^T q_h meets the latents directly, and because the softmax weights are scalars the
// value map is applied once to the weighted sum of latents.  What is left for this kernel is attention with one
// shared "head" of width `rank` whose keys and values are the same rows:
//
//     out[b, h] = gate[b, h] * sum_j softmax_j(scale * q'[b, h] . c_j) c_j        (all j < ctx_len)
//
// A page [16, rank] is fetched once for all heads and serves as K and as V: rank * 2 bytes per token.
//
//   grid     (batch x head groups of 16 * MT, splits): the head groups of a row are neighbours, so the second finds the
//            row's pages in L2
//   load     tiles of tokens by TMA (boxes of 16 tokens x 128 B, 128-byte swizzle, one box per lane of warp 0) into a ring
//            of stages; a stage is refilled right after the barrier that every warp reaches only when it is done with the
//            tile before, so no "empty" barriers and no producer warp are needed
//   scores   the groups of 8 tokens of a tile are dealt to the warps; S[heads x 8 tokens] over the whole rank by mma.sync
//            m16n8k16.  The projected queries stay in registers, or in shared memory where they do not fit.
//   softmax  exponentials in fp32 against the common running maximum; the warps' row maxima meet in shared memory, P in
//            bf16 goes to shared memory
//   values   warp w owns rank / warps columns of the output: O += P C over the tile's tokens
//   None of the units is near its limit here - what costs is the chain score -> maximum -> exponential -> value with two
//   barriers per tile -, so two CTAs of four warps share an SM where registers and shared memory allow.  (A loop skewed by
//   one tile, with the next tile's scores ahead of a single barrier, was slower: it needs every tile one step earlier, and
//   the ring is only three tiles deep.)
//   out      as in paged_attn.cu: bf16 straight from registers when the row fits one split, else fp32 partials that
//            a second kernel folds in split order.
// Every wait is bounded.

#include "common.cuh"
#include "host.h"

namespace b200 {

constexpr int kLatPage = 16;

// R: rank.  MT: head tiles of 16 per CTA.  WARPS: each owns R / WARPS columns of the output.  TILE: tokens per pipeline
// stage.  CTAS: CTAs per SM aimed for.
template <int R_, int MT_, int WARPS_, int TILE_, int STAGES_, int CTAS_>
struct LatentCfg {
  static constexpr int R = R_, MT = MT_, kWarps = WARPS_, kTile = TILE_, kStages = STAGES_, kCtas = CTAS_;
  static constexpr int kPages = kTile / kLatPage;
  static constexpr int kHalf = kTile * 128;  // 64 columns of a tile
  static constexpr int kHalves = R / 64;
  static constexpr bool kQRegs = R * MT <= 512;
  static constexpr int kStageBytes = kHalves * kHalf;
  static constexpr int kQBytes = kQRegs ? 0 : MT * 16 * R * 2;
  static constexpr int kPBytes = MT * 16 * 128;
  static constexpr int kRedBytes = kWarps * MT * 16 * 4;
  static constexpr int kSmemBytes = 1024 + kStages * kStageBytes + kQBytes + kPBytes + kRedBytes + 8 * kStages;
  static constexpr int kThreads = kWarps * 32;
  static_assert(kPages * kHalves <= 32, "one TMA box per lane");
  static_assert(!kQRegs || MT * 16 * R * 2 <= kStageBytes, "the queries pass through the last stage");

  static_assert(kTile <= 64 && kTile % 16 == 0 && R % (kWarps * 16) == 0, "tile shape");
};

template <class Cfg>
__global__ void __launch_bounds__(Cfg::kThreads, Cfg::kCtas)
latent_attn_decode_kernel(const __grid_constant__ CUtensorMap c_map, const __nv_bfloat16* __restrict__ q,
                          const int* __restrict__ block_table, const int* __restrict__ ctx_lens,
                          float* __restrict__ part_o, float2* __restrict__ part_ml, __nv_bfloat16* __restrict__ out,
                          int* __restrict__ err, int heads, int num_blocks, int max_pages, int split_tokens,
                          int max_splits, float scale_log2, const float* __restrict__ gate, int head_groups) {
#ifdef B200_DEVICE_OK
  grid_dep_wait();
  grid_dep_launch();
  constexpr int R = Cfg::R, MT = Cfg::MT, NW = Cfg::kWarps, STAGES = Cfg::kStages;
  constexpr int kLatTile = Cfg::kTile, kLatHalf = Cfg::kHalf, kLatPages = Cfg::kPages, kHalves = Cfg::kHalves;
  constexpr int kCols = R / NW, kNt = kCols / 8;  // output columns of a warp, n tiles of 8
  extern __shared__ uint8_t smem_raw[];
  const uint32_t ring = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (ring - smem_u32(smem_raw));
  const uint32_t p_sm = ring + STAGES * Cfg::kStageBytes + Cfg::kQBytes;
  uint8_t* p_ptr = base_ptr + STAGES * Cfg::kStageBytes + Cfg::kQBytes;
  float* red = reinterpret_cast<float*>(p_ptr + Cfg::kPBytes);  // [NW][MT * 16]
  const uint32_t bars = p_sm + Cfg::kPBytes + Cfg::kRedBytes;   // full[STAGES]

  const int b = blockIdx.x / head_groups, split = blockIdx.y, h0 = (blockIdx.x - b * head_groups) * (16 * MT);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int L = ctx_lens[b];
  if (L < 0 || L > max_pages * kLatPage) {
    if (threadIdx.x == 0) set_error(err, kErrDevBadCtxLen);
    L = L < 0 ? 0 : max_pages * kLatPage;
  }
  const int start = split * split_tokens;
  if (start >= L) {  // uniform for the whole CTA
    if (L == 0 && split == 0)
      for (int i = threadIdx.x; i < min(16 * MT, heads - h0) * R; i += blockDim.x)
        out[(static_cast<size_t>(b) * heads + h0) * R + i] = __float2bfloat16(0.f);
    return;
  }
  const int end = min(L, start + split_tokens);
  const int n_tiles = (end - start + kLatTile - 1) / kLatTile;
  const int first_page = start / kLatPage, last_page = (end - 1) / kLatPage;

  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) mbar_init(bars + 8 * s, 1);
    fence_mbar_init();
    fence_proxy_async();
  }
  // projected queries to shared memory, [64-column half][head][128 B] swizzled: to stay there, or on their way to registers
  // in the last stage, which the first tiles do not use
  constexpr uint32_t kQOff = Cfg::kQRegs ? (STAGES - 1) * Cfg::kStageBytes : STAGES * Cfg::kStageBytes;
  for (int i = threadIdx.x; i < MT * 16 * (R / 8); i += blockDim.x) {
    const int row = i / (R / 8), ch = i % (R / 8);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h0 + row < heads)
      v = *reinterpret_cast<const uint4*>(q + (static_cast<size_t>(b) * heads + h0 + row) * R + ch * 8);
    *reinterpret_cast<uint4*>(base_ptr + kQOff + (ch >> 3) * (MT * 16 * 128) + swz128(row, ch & 7)) = v;
  }
  __syncthreads();

  // ---------------------------------------------------------------- loads --
  // Lane of warp 0 -> one box of a tile.  The page id of the next tile to load is fetched one step ahead.  Pages past the
  // split's end hold nothing that may be read; the last valid page stands in (its scores are masked).
  const int* table_row = block_table + static_cast<size_t>(b) * max_pages;
  const int pg = lane / kHalves, half = lane % kHalves;
  const bool issuer = warp == 0 && lane < kLatPages * kHalves;
  int next_id = 0;
  auto fetch_id = [&](int tile) {
    if (issuer) next_id = table_row[min(first_page + tile * kLatPages + pg, last_page)];
  };
  auto load_tile = [&](int tile) {  // whole warp 0
    int id = next_id;
    if (id < 0 || id >= num_blocks) {
      set_error(err, kErrDevBadBlockId);
      id = 0;
    }
    const int slot = tile % STAGES;
    if (lane == 0) mbar_arrive_expect_tx(bars + 8 * slot, Cfg::kStageBytes);
    __syncwarp();
    if (issuer)
      tma_load_2d(ring + slot * Cfg::kStageBytes + half * kLatHalf + pg * (kLatPage * 128), &c_map, bars + 8 * slot,
                  half * 64, id * kLatPage);
  };
  if (warp == 0) {
    for (int t = 0; t < min(STAGES - 1, n_tiles); ++t) {
      fetch_id(t);
      load_tile(t);
    }
    fetch_id(STAGES - 1);
  }

  // ----------------------------------------------------------------- math --
  const int gq = lane >> 2, tq = lane & 3, lj = lane >> 3, lr = lane & 7;
  const int v_tok = (lj & 1) * 8 + lr, v_sub = lj >> 1;
  uint32_t qa[Cfg::kQRegs ? MT : 1][Cfg::kQRegs ? R / 16 : 1][4];
  auto q_frag = [&](int mt, int ks, uint32_t (&a)[4]) {
    const int c = ks * 2 + (lj >> 1);
    ldmatrix_x4(ring + kQOff + (c >> 3) * (MT * 16 * 128) + swz128(mt * 16 + (lj & 1) * 8 + lr, c & 7), a[0], a[1], a[2], a[3]);
  };
  if (Cfg::kQRegs) {
#pragma unroll
    for (int mt = 0; mt < (Cfg::kQRegs ? MT : 1); ++mt)
#pragma unroll
      for (int ks = 0; ks < (Cfg::kQRegs ? R / 16 : 1); ++ks) q_frag(mt, ks, qa[mt][ks]);
    fence_proxy_async();  // read before the copies that will refill the stage (ordered by the loop's first barrier)
  }
  float o[MT][kNt][4];
  float m_run[MT][2], l_run[MT][2];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
    for (int n = 0; n < kNt; ++n) o[mt][n][0] = o[mt][n][1] = o[mt][n][2] = o[mt][n][3] = 0.f;
    m_run[mt][0] = m_run[mt][1] = -INFINITY;
    l_run[mt][0] = l_run[mt][1] = 0.f;
  }
  constexpr int kGroups = kLatTile / 8;                  // groups of 8 tokens, dealt to the warps
  constexpr int kMine = (kGroups + NW - 1) / NW;         // per warp (some warps may have one less)
  constexpr int kChains = MT == 1 && R % 64 == 0 ? 4 : 2;  // independent accumulators: short chains of dependent MMAs
  bool alive = true;
  float s[kMine][MT][4];
  auto wait_tile = [&](int t) {
    if (alive) alive = mbar_wait(bars + 8 * (t % STAGES), (t / STAGES) & 1, err);
  };
  // scores of tile t into s (log2 domain), this warp's row maxima to shared memory
  auto score = [&](int t) {
    const uint32_t cbase = ring + (t % STAGES) * Cfg::kStageBytes;
    const int left = end - (start + t * kLatTile);  // tokens of the tile that exist
    float mx[MT][2];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) mx[mt][0] = mx[mt][1] = -INFINITY;
#pragma unroll
    for (int g = 0; g < kMine; ++g) {
      const int n8 = warp + g * NW;
      float acc[kChains][MT][4];
#pragma unroll
      for (int e = 0; e < kChains; ++e)
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) acc[e][mt][0] = acc[e][mt][1] = acc[e][mt][2] = acc[e][mt][3] = 0.f;
      if (n8 < kGroups) {
#pragma unroll
        for (int kk = 0; kk < R / 32; ++kk) {  // 32 latent columns: two k steps
          uint32_t b0, b1, b2, b3;
          const int ch = kk * 4 + lj;
          ldmatrix_x4(cbase + (ch >> 3) * kLatHalf + swz128(n8 * 8 + lr, ch & 7), b0, b1, b2, b3);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            if (Cfg::kQRegs) {
              mma_bf16_16816(acc[(2 * kk) % kChains][mt], qa[Cfg::kQRegs ? mt : 0][Cfg::kQRegs ? 2 * kk : 0], b0, b1);
              mma_bf16_16816(acc[(2 * kk + 1) % kChains][mt], qa[Cfg::kQRegs ? mt : 0][Cfg::kQRegs ? 2 * kk + 1 : 0], b2, b3);
            } else {
              uint32_t a[4], a2[4];
              q_frag(mt, 2 * kk, a);
              q_frag(mt, 2 * kk + 1, a2);
              mma_bf16_16816(acc[(2 * kk) % kChains][mt], a, b0, b1);
              mma_bf16_16816(acc[(2 * kk + 1) % kChains][mt], a2, b2, b3);
            }
          }
        }
      }
      const int tok = n8 * 8 + 2 * tq;
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const bool seen = n8 < kGroups && tok + (e & 1) < left;
          float sum = acc[0][mt][e] + acc[1][mt][e];
          if (kChains == 4) sum += acc[kChains - 2][mt][e] + acc[kChains - 1][mt][e];
          s[g][mt][e] = seen ? sum * scale_log2 : -INFINITY;
        }
        mx[mt][0] = fmaxf(mx[mt][0], fmaxf(s[g][mt][0], s[g][mt][1]));
        mx[mt][1] = fmaxf(mx[mt][1], fmaxf(s[g][mt][2], s[g][mt][3]));
      }
    }
    float* mine = red + warp * (MT * 16);
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        float v = mx[mt][hf];
        v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
        v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
        if (tq == 0) mine[mt * 16 + hf * 8 + gq] = v;
      }
  };
#pragma unroll 1
  for (int i = 0; i < n_tiles; ++i) {
    wait_tile(i);
    score(i);
    // every warp's maxima are written, and every warp is done with the P and the latents of the tile before
    __syncthreads();
    if (warp == 0 && i + STAGES - 1 < n_tiles) {
      load_tile(i + STAGES - 1);
      fetch_id(i + STAGES);
    }
    const uint32_t cbase = ring + (i % STAGES) * Cfg::kStageBytes;
    float alpha[MT][2];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        float v = m_run[mt][hf];
#pragma unroll
        for (int w = 0; w < NW; ++w) v = fmaxf(v, red[w * (MT * 16) + mt * 16 + hf * 8 + gq]);
        alpha[mt][hf] = exp2f(m_run[mt][hf] - v);  // every tile has a token, so v is finite
        m_run[mt][hf] = v;
        l_run[mt][hf] *= alpha[mt][hf];
      }
#pragma unroll
    for (int g = 0; g < kMine; ++g) {
      const int n8 = warp + g * NW;
      if (n8 < kGroups) {
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
          for (int hf = 0; hf < 2; ++hf) {
            const float p0 = exp2f(s[g][mt][2 * hf] - m_run[mt][hf]), p1 = exp2f(s[g][mt][2 * hf + 1] - m_run[mt][hf]);
            l_run[mt][hf] += p0 + p1;
            *reinterpret_cast<uint32_t*>(p_ptr + swz128(mt * 16 + hf * 8 + gq, n8) + tq * 4) = pack_bf16x2(p0, p1);
          }
      }
    }
    __syncthreads();  // P is complete
    bool resc = false;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) resc = resc || alpha[mt][0] != 1.f || alpha[mt][1] != 1.f;
    if (__any_sync(0xffffffffu, resc)) {
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < kNt; ++n) {
          o[mt][n][0] *= alpha[mt][0];
          o[mt][n][1] *= alpha[mt][0];
          o[mt][n][2] *= alpha[mt][1];
          o[mt][n][3] *= alpha[mt][1];
        }
    }
#pragma unroll
    for (int ks = 0; ks < kLatTile / 16; ++ks) {
      uint32_t pa[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
        ldmatrix_x4(p_sm + swz128(mt * 16 + (lj & 1) * 8 + lr, ks * 2 + (lj >> 1)), pa[mt][0], pa[mt][1], pa[mt][2], pa[mt][3]);
#pragma unroll
      for (int np = 0; np < kNt / 2; ++np) {
        uint32_t v0, v1, v2, v3;
        const int ch = warp * (kCols / 8) + np * 2 + v_sub;
        ldmatrix_x4_trans(cbase + (ch >> 3) * kLatHalf + swz128(ks * 16 + v_tok, ch & 7), v0, v1, v2, v3);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16_16816(o[mt][2 * np], pa[mt], v0, v1);
          mma_bf16_16816(o[mt][2 * np + 1], pa[mt], v2, v3);
        }
      }
    }
  }

  // normalisers: each warp has the sums over its own tokens
  __syncthreads();
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      float v = l_run[mt][hf];
      v += __shfl_xor_sync(0xffffffffu, v, 1);
      v += __shfl_xor_sync(0xffffffffu, v, 2);
      if (tq == 0) red[warp * (MT * 16) + mt * 16 + hf * 8 + gq] = v;
    }
  __syncthreads();
  const int nsplits = (L + split_tokens - 1) / split_tokens;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      float l = 0.f;
#pragma unroll
      for (int w = 0; w < NW; ++w) l += red[w * (MT * 16) + mt * 16 + hf * 8 + gq];
      const int h = h0 + mt * 16 + hf * 8 + gq;
      if (h >= heads) continue;
      const size_t row = static_cast<size_t>(b) * heads + h;
      if (nsplits == 1) {
        const float inv = head_gate(gate, row) / l;
        __nv_bfloat16* od = out + row * R + warp * kCols + 2 * tq;
#pragma unroll
        for (int n = 0; n < kNt; ++n)
          *reinterpret_cast<uint32_t*>(od + n * 8) = pack_bf16x2(o[mt][n][2 * hf] * inv, o[mt][n][2 * hf + 1] * inv);
      } else {
        const size_t prow = row * max_splits + split;
        float* od = part_o + prow * R + warp * kCols + 2 * tq;
#pragma unroll
        for (int n = 0; n < kNt; ++n)
          *reinterpret_cast<float2*>(od + n * 8) = make_float2(o[mt][n][2 * hf], o[mt][n][2 * hf + 1]);
        if (warp == 0 && tq == 0) part_ml[prow] = make_float2(m_run[mt][hf], l);
      }
    }
#endif
}

// Folds the split partials of one (row, head) in split order: one CTA per row, four columns per thread.
__global__ void __launch_bounds__(128)
latent_attn_reduce_kernel(const float* __restrict__ part_o, const float2* __restrict__ part_ml,
                          const int* __restrict__ ctx_lens, __nv_bfloat16* __restrict__ out, int heads, int rank,
                          int max_splits, int split_tokens, int max_ctx, const float* __restrict__ gate) {
  grid_dep_wait();
  grid_dep_launch();
  const size_t row = blockIdx.x;
  int L = ctx_lens[blockIdx.x / heads];
  L = L < 0 ? 0 : (L > max_ctx ? max_ctx : L);
  const int n = (L + split_tokens - 1) / split_tokens;
  const int col = threadIdx.x * 4;
  if (n <= 1 || col >= rank) return;
  const float2* ml = part_ml + row * max_splits;
  const float* po = part_o + row * max_splits * rank + col;
  float m = -INFINITY;
  for (int s = 0; s < n; ++s) m = fmaxf(m, ml[s].x);
  float den = 0.f;
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
  for (int s = 0; s < n; ++s) {
    const float w = exp2f(ml[s].x - m);
    const float4 v = *reinterpret_cast<const float4*>(po + static_cast<size_t>(s) * rank);
    den += w * ml[s].y;
    acc.x += w * v.x;
    acc.y += w * v.y;
    acc.z += w * v.z;
    acc.w += w * v.w;
  }
  const float inv = head_gate(gate, row) / den;
  uint2 r;
  r.x = pack_bf16x2(acc.x * inv, acc.y * inv);
  r.y = pack_bf16x2(acc.z * inv, acc.w * inv);
  *reinterpret_cast<uint2*>(out + row * rank + col) = r;
}

template <class Cfg>
static int launch_latent(const void* q, const void* c_pool, const int* block_table, const int* ctx_lens, void* out,
                         const AttnWorkspace& w, int batch, int heads, int num_blocks, int max_pages, float scale,
                         int split_tokens, int max_splits, const float* gate, cudaStream_t st) {
  static_assert(Cfg::kSmemBytes <= 232448, "more shared memory than a CTA may have");
  CUtensorMap cmap;
  int rc = get_tensor_map_2d(c_pool, static_cast<uint64_t>(num_blocks) * kLatPage, Cfg::R, 2, kLatPage, 64, &cmap);
  if (rc) return rc;
  rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&latent_attn_decode_kernel<Cfg>), Cfg::kSmemBytes);
  if (rc) return rc;
  const int head_groups = (heads + 16 * Cfg::MT - 1) / (16 * Cfg::MT);
  const dim3 grid(batch * head_groups, max_splits);
  B200_CUDA(launch_overlapped(latent_attn_decode_kernel<Cfg>, grid, dim3(Cfg::kThreads), Cfg::kSmemBytes, st, cmap,
                              static_cast<const __nv_bfloat16*>(q), block_table, ctx_lens, w.o, w.ml,
                              static_cast<__nv_bfloat16*>(out), w.err, heads, num_blocks, max_pages, split_tokens,
                              max_splits, scale * 1.4426950408889634f, gate, head_groups));
  if (max_splits > 1)
    B200_CUDA(launch_overlapped(latent_attn_reduce_kernel, dim3(batch * heads), dim3(128), 0, st, w.o, w.ml, ctx_lens,
                                static_cast<__nv_bfloat16*>(out), heads, Cfg::R, max_splits, split_tokens,
                                max_pages * kLatPage, gate));
  return 0;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_latent_attn_supported(int rank, int page_size) {
  return page_size == kLatPage && (rank == 64 || rank == 128 || rank == 192 || rank == 256 || rank == 384 || rank == 512);
}

extern "C" int b200_latent_attn_decode(const void* q, const void* c_pool, const int32_t* block_table,
                                       const int32_t* ctx_lens, void* out, void* workspace, size_t workspace_bytes,
                                       int batch, int num_heads, int rank, int page_size, int num_blocks,
                                       int max_pages_per_seq, float scale, int split_tokens, const float* gate,
                                       void* stream) {
  B200_REQUIRE(q && c_pool && block_table && ctx_lens && out && workspace, "latent_attn_decode: null pointer");
  B200_REQUIRE(batch > 0 && num_heads > 0 && num_blocks > 0 && max_pages_per_seq > 0,
               "latent_attn_decode: non-positive dimension");
  B200_REQUIRE(b200_latent_attn_supported(rank, page_size), "latent_attn_decode: rank %d, page %d", rank, page_size);
  B200_REQUIRE(split_tokens > 0 && split_tokens % kLatPage == 0, "latent_attn_decode: split_tokens %d not a multiple of %d",
               split_tokens, kLatPage);
  B200_REQUIRE(((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(c_pool) |
                 reinterpret_cast<uintptr_t>(out)) & 15) == 0,
               "latent_attn_decode: buffers must be 16-byte aligned");
  int rc = check_device(nullptr);
  if (rc) return rc;
  const int ms = (max_pages_per_seq * kLatPage + split_tokens - 1) / split_tokens;
  B200_REQUIRE(ms <= 65535, "latent_attn_decode: grid too large");
  AttnWorkspace w = carve(workspace, batch, num_heads, rank, ms);
  if (workspace_bytes < w.bytes) {
    set_detail("latent_attn_decode: workspace %zu < required %zu", workspace_bytes, w.bytes);
    return -kErrWorkspace;
  }
  cudaStream_t st = as_stream(stream);
#define B200_LAT_ARGS q, c_pool, block_table, ctx_lens, out, w, batch, num_heads, num_blocks, max_pages_per_seq, scale, \
                      split_tokens, ms, gate, st
  //                    rank MT warps tile stages CTAs
  const bool two = num_heads > 16;
  switch (rank) {
    case 64: return two ? launch_latent<LatentCfg<64, 2, 1, 64, 4, 3>>(B200_LAT_ARGS)
                        : launch_latent<LatentCfg<64, 1, 1, 64, 4, 3>>(B200_LAT_ARGS);
    case 128: return two ? launch_latent<LatentCfg<128, 2, 2, 64, 4, 3>>(B200_LAT_ARGS)
                         : launch_latent<LatentCfg<128, 1, 2, 64, 4, 3>>(B200_LAT_ARGS);
    case 192: return two ? launch_latent<LatentCfg<192, 2, 3, 48, 4, 2>>(B200_LAT_ARGS)
                         : launch_latent<LatentCfg<192, 1, 3, 48, 4, 2>>(B200_LAT_ARGS);
    case 256: return two ? launch_latent<LatentCfg<256, 2, 4, 64, 3, 2>>(B200_LAT_ARGS)
                         : launch_latent<LatentCfg<256, 1, 4, 64, 3, 2>>(B200_LAT_ARGS);
    case 384: return two ? launch_latent<LatentCfg<384, 2, 6, 48, 4, 1>>(B200_LAT_ARGS)
                         : launch_latent<LatentCfg<384, 1, 3, 32, 4, 2>>(B200_LAT_ARGS);
    default: return two ? launch_latent<LatentCfg<512, 2, 4, 32, 2, 2>>(B200_LAT_ARGS)
                        : launch_latent<LatentCfg<512, 1, 4, 32, 3, 2>>(B200_LAT_ARGS);
  }
#undef B200_LAT_ARGS
}
