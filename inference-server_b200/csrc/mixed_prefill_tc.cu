// Attention with mixed heads (see mixed_attn.cu) for a chunk of prompt tokens of one sequence on the tcgen05 tensor cores:
// bf16, key size a multiple of 64 per kv head, value size 64, 128, 192 or 256, up to 128 query heads per kv head.
//
//   grid     (query tiles, kv heads).  A CTA owns 128 score rows: 128 / per consecutive positions x the `per` query heads of
//            its kv head, and walks the key tiles (128 keys = 8 pages) from the one that holds the first key its first row
//            sees to the one of its last position.
//   warp 0   K producer: a tile's keys of ALL kv heads, 64 columns (16 KiB: 8 boxes of 16 tokens x 128 B) at a time, into a
//            ring.  Before that the mixed queries of the tile, once, if its boxes fit the swizzle (per a multiple of 8).
//   warp 1   issuer (one thread): S(0), then S(j + 1) and O += P(j) V(j) for every tile j.  S = Q' K^T is 4 x tcgen05.mma
//            M128 N128 K16 per 64 columns into one of two S accumulators in TMEM; P (bf16) is an A operand in TMEM, V an
//            MN-major B operand straight from its page layout.  While the softmax of tile j runs, S(j + 1) is in the tensor pipe.
//   warp 2   the distance table: per tile the slice of B[h][.] that the tile's rows and keys meet, as +inf where a distance is
//            negative (a later token) or outside the window, so the mask costs nothing of its own.
//   warp 3   V producer: the values of the CTA's kv head, one tile at a time.
//   warps 4-11  softmax: a thread owns a score row and 64 of the tile's 128 keys (TMEM lanes are bound to warp_id % 4; the two
//            warps with the same rows meet on a named barrier for the row maximum).  s = score * log2 e - B from the slice in
//            shared memory, lazy rescale of O as in paged_prefill_tc.cu, P = exp2(s - m) stored to TMEM.
//
// TMEM: S0 columns 0-127, S1 128-255, O from 256 on, P in the last 64 columns; with value size 256, where none are left, P(j)
// lies over S(j), and the issuer then waits for the product with P(j) before it writes that S accumulator again.
// Every mbarrier wait is bounded; one that runs out records kErrDevWaitTimeout, and the thread stops waiting but keeps the loop
// structure (the named barriers between partner warps are still met), so the kernel ends.

#include "glue.cuh"

namespace b200 {

constexpr int kMpPage = 16;
constexpr int kMpRows = 128, kMpKeys = 128;
constexpr int kMpChunk = 128 * 128;  // 128 rows x 64 bf16
constexpr int kMpSoftmaxWarps = 8;
constexpr int kMpThreads = (4 + kMpSoftmaxWarps) * 32;
constexpr int kMpMaxStages = 8;
constexpr float kMpRescaleLog2 = 8.f;
constexpr float kMpLog2e = 1.4426950408889634f;

struct MixedPrefillParams {
  const int* table_row;
  const __nv_bfloat16* q;  // [tokens, heads, k_chunks * 64]
  const float* bias;       // [heads, bias_ld]
  __nv_bfloat16* out;      // [tokens, out_ld]
  int* err;
  int bias_ld, window, out_ld;
  float out_scale;
  int num_tokens, first_pos, heads, kv_heads, num_blocks;
  int k_chunks;            // 64-wide pieces of a mixed query (all kv heads)
  int dk_chunks;           // of one kv head's keys
  int stages, q_tma;
  int bias_stride;         // floats per head of a slice
};

__host__ __device__ constexpr uint32_t mp_idesc(uint32_t n, uint32_t b_mn) {
  return (1u << 4) | (1u << 7) | (1u << 10) | (b_mn << 16) | ((n >> 3) << 17) | ((128u >> 4) << 24);
}
__device__ __forceinline__ void mp_mma_ss(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}" ::"r"(d), "l"(a), "l"(b), "r"(idesc), "r"(acc)
      : "memory");
}
// A from TMEM: lane = row, a 32-bit column = two neighbouring K elements.
__device__ __forceinline__ void mp_mma_ts(uint32_t d, uint32_t a, uint64_t b, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}" ::"r"(d), "r"(a), "l"(b), "r"(idesc), "r"(acc)
      : "memory");
}
__device__ __forceinline__ uint64_t mp_desc_mn(uint32_t addr) {  // MN-major, 128-byte swizzle, next 64 columns kMpChunk further
  uint64_t d = 0;
  d |= static_cast<uint64_t>((addr & 0x3FFFFu) >> 4);
  d |= static_cast<uint64_t>(kMpChunk >> 4) << 16;
  d |= static_cast<uint64_t>(1024 >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
__device__ __forceinline__ void mp_tmem_st32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16,"
      "%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31,%32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]),
        "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]),
        "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}
__device__ __forceinline__ void mp_tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ float mp_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void mp_pair_barrier(int quarter) {
  switch (quarter) {
    case 0: asm volatile("bar.sync 1, 64;" ::: "memory"); break;
    case 1: asm volatile("bar.sync 2, 64;" ::: "memory"); break;
    case 2: asm volatile("bar.sync 3, 64;" ::: "memory"); break;
    default: asm volatile("bar.sync 4, 64;" ::: "memory"); break;
  }
}

template <int DV>
__global__ void __launch_bounds__(kMpThreads, 1)
mixed_prefill_tc_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map,
                        const __grid_constant__ CUtensorMap v_map, const MixedPrefillParams p) {
#ifdef B200_DEVICE_OK
  constexpr int kVChunks = DV / 64;
  constexpr bool kAlias = DV > 192;  // P over S
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
  const uint32_t q_sm = base, v_sm = q_sm + p.k_chunks * kMpChunk, k_sm = v_sm + kVChunks * kMpChunk;
  uint8_t* extra = base_ptr + (p.k_chunks + kVChunks + p.stages) * kMpChunk;
  const uint32_t bars = k_sm + p.stages * kMpChunk;
  const uint32_t bar_q = bars, bar_vfull = bars + 8, bar_vempty = bars + 16;
  const uint32_t bar_sfull = bars + 24, bar_sempty = bars + 40;  // [2] each
  const uint32_t bar_pfull = bars + 56, bar_odone = bars + 64;
  const uint32_t bar_bfull = bars + 72, bar_bempty = bars + 88;  // [2] each: slice of the distance table
  const uint32_t bar_kfull = bars + 104, bar_kempty = bar_kfull + 8 * kMpMaxStages;
  uint32_t* tmem_base_sm = reinterpret_cast<uint32_t*>(extra + 240);
  float* mx_sm = reinterpret_cast<float*>(extra + 256);  // [2 tiles][2 halves][128 rows]
  float* l_sm = mx_sm + 2 * 2 * kMpRows;                 // [2 halves][128 rows]
  float* b_sm = l_sm + 2 * kMpRows;                      // [2][per][bias_stride]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per = p.heads / p.kv_heads, QT = kMpRows / per;
  if (threadIdx.x == 32) {
    tma_prefetch_desc(&q_map);
    tma_prefetch_desc(&k_map);
    tma_prefetch_desc(&v_map);
  }
  if (threadIdx.x == 0) {
    mbar_init(bar_q, p.q_tma ? 1 : kMpSoftmaxWarps);
    mbar_init(bar_vfull, 1);
    mbar_init(bar_vempty, 1);
    mbar_init(bar_pfull, kMpSoftmaxWarps);
    mbar_init(bar_odone, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(bar_sfull + 8 * s, 1);
      mbar_init(bar_sempty + 8 * s, kMpSoftmaxWarps);
      mbar_init(bar_bfull + 8 * s, 1);
      mbar_init(bar_bempty + 8 * s, kMpSoftmaxWarps);
    }
    for (int s = 0; s < p.stages; ++s) {
      mbar_init(bar_kfull + 8 * s, 1);
      mbar_init(bar_kempty + 8 * s, 1);
    }
    fence_mbar_init();
    fence_proxy_async();
  }
  if (warp == 1) tmem_alloc(smem_u32(tmem_base_sm), 512);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_base_sm;
  grid_dep_wait();
  grid_dep_launch();

  const int qt = static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x);  // late positions first
  const int g = blockIdx.y, t0 = qt * QT;
  const int t_end = min(t0 + QT, p.num_tokens);
  const int p0 = p.first_pos + t0, last_pos = p.first_pos + t_end - 1;
  const int kt0 = max(0, p0 - p.window + 1) / kMpKeys;
  const int n_tiles = last_pos / kMpKeys - kt0 + 1;
  const int last_page = last_pos / kMpPage;

  if (warp == 0 || warp == 3) {
    // -------------------------------------------------------- K / V producers ------
    if (warp == 0 && p.q_tma) {
      if (lane == 0) mbar_arrive_expect_tx(bar_q, p.k_chunks * kMpChunk);
      __syncwarp();
      for (int i = lane; i < p.k_chunks * QT; i += 32) {
        const int tl = i / p.k_chunks, c = i - tl * p.k_chunks;
        tma_load_2d(q_sm + c * kMpChunk + tl * per * 128, &q_map, bar_q, c * 64, (t0 + tl) * p.heads + g * per);
      }
    }
    bool alive = true;
    uint32_t it = 0;
#pragma unroll 1
    for (int j = 0; j < n_tiles && alive; ++j) {
      // lanes 0-7 own a page each; pages past the last position stand in for by it: their keys are masked, their values meet
      // weights of 0
      int page = 0;
      if (lane < 8) {
        page = __ldg(p.table_row + min((kt0 + j) * 8 + lane, last_page));
        if (page < 0 || page >= p.num_blocks) {
          set_error(p.err, kErrDevBadBlockId);
          page = 0;
        }
      }
      const int row0 = page * p.kv_heads * kMpPage;
      if (warp == 0) {
#pragma unroll 1
        for (int c = 0; c < p.k_chunks && alive; ++c, ++it) {
          const uint32_t st = it % p.stages, ph = (it / p.stages) & 1;
          alive = mbar_wait(bar_kempty + 8 * st, ph ^ 1, p.err);
          alive = __all_sync(0xffffffffu, alive);
          if (!alive) break;
          if (lane == 0) mbar_arrive_expect_tx(bar_kfull + 8 * st, kMpChunk);
          __syncwarp();
          const int head = c / p.dk_chunks;
          if (lane < 8)
            tma_load_2d(k_sm + st * kMpChunk + lane * (kMpPage * 128), &k_map, bar_kfull + 8 * st, (c - head * p.dk_chunks) * 64,
                        row0 + head * kMpPage);
        }
      } else {
        alive = mbar_wait(bar_vempty, (j & 1) ^ 1, p.err);
        alive = __all_sync(0xffffffffu, alive);
        if (!alive) break;
        if (lane == 0) mbar_arrive_expect_tx(bar_vfull, kVChunks * kMpChunk);
        __syncwarp();
        if (lane < 8)
#pragma unroll
          for (int c = 0; c < kVChunks; ++c)
            tma_load_2d(v_sm + c * kMpChunk + lane * (kMpPage * 128), &v_map, bar_vfull, c * 64, row0 + g * kMpPage);
      }
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- issuer ------
    if (lane == 0) {
      constexpr uint32_t idesc_s = mp_idesc(kMpKeys, 0), idesc_o = mp_idesc(DV, 1);
      const uint32_t tmem_o = tmem_base + 256;
      bool alive = mbar_wait(bar_q, 0, p.err);
      uint32_t it = 0;
      auto scores = [&](int t) {
        const int sb = t & 1;
        const uint32_t ph = (t >> 1) & 1;
        if (alive) alive = mbar_wait(bar_sempty + 8 * sb, ph ^ 1, p.err);
        if (kAlias && t >= 2 && alive) alive = mbar_wait(bar_odone, (t - 2) & 1, p.err);  // P(t - 2) lies there
#pragma unroll 1
        for (int c = 0; c < p.k_chunks && alive; ++c, ++it) {
          const uint32_t st = it % p.stages;
          alive = mbar_wait(bar_kfull + 8 * st, (it / p.stages) & 1, p.err);
          if (!alive) break;
          tc_fence_after();
          const uint64_t a0 = umma_desc_k128(q_sm + c * kMpChunk), b0 = umma_desc_k128(k_sm + st * kMpChunk);
#pragma unroll
          for (int k = 0; k < 4; ++k)
            mp_mma_ss(tmem_base + sb * kMpKeys, a0 + 2 * k, b0 + 2 * k, idesc_s, (c > 0 || k > 0) ? 1u : 0u);
          tc_commit(bar_kempty + 8 * st);
        }
        if (alive) tc_commit(bar_sfull + 8 * sb);
      };
      scores(0);
#pragma unroll 1
      for (int j = 0; j < n_tiles && alive; ++j) {
        if (j + 1 < n_tiles) scores(j + 1);
        if (alive) alive = mbar_wait(bar_vfull, j & 1, p.err);
        if (alive) alive = mbar_wait(bar_pfull, j & 1, p.err);
        if (!alive) break;
        tc_fence_after();
        const uint32_t pa = tmem_base + (kAlias ? static_cast<uint32_t>((j & 1) * kMpKeys) : 448u);
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          mp_mma_ts(tmem_o, pa + kk * 8, mp_desc_mn(v_sm + kk * (16 * 128)), idesc_o, (j > 0 || kk > 0) ? 1u : 0u);
        tc_commit(bar_odone);
        tc_commit(bar_vempty);
      }
    }
  } else if (warp == 2) {
    // ------------------------------------------- slices of the distance table ------
    // entry x of a head: distance p0 - (first key of the tile) - 127 + x
    bool alive = true;
    const int span = kMpKeys + QT - 1;
#pragma unroll 1
    for (int j = 0; j < n_tiles && alive; ++j) {
      alive = mbar_wait(bar_bempty + 8 * (j & 1), ((j >> 1) & 1) ^ 1, p.err);
      alive = __all_sync(0xffffffffu, alive);
      if (!alive) break;
      const int d0 = p0 - (kt0 + j) * kMpKeys - (kMpKeys - 1);
      float* dst = b_sm + (j & 1) * per * p.bias_stride;
      for (int hh = 0; hh < per; ++hh) {
        const float* src = p.bias + static_cast<size_t>(g * per + hh) * p.bias_ld;
#pragma unroll 4
        for (int x = lane; x < span; x += 32) {
          const int d = d0 + x;
          dst[hh * p.bias_stride + x] = d >= 0 && d < p.window && d < p.bias_ld ? __ldg(src + d) * kMpLog2e : INFINITY;
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_bfull + 8 * (j & 1));
    }
  } else {
    // --------------------------------------------------------------- softmax ------
    const int sw = warp - 4, hf = sw >> 2, quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(quarter * 32) << 16);
    const uint32_t tmem_o = lane_addr + 256 + hf * (DV / 2);
    const int tl = r / per, head = r - tl * per;
    const bool real = tl < QT && t0 + tl < p.num_tokens;
    if (!p.q_tma) {  // copy the Q' tile: neighbouring threads take neighbouring 16-byte pieces of a row
      const int pieces = p.k_chunks * 8;
      for (int i = sw * 32 + lane; i < kMpRows * pieces; i += kMpSoftmaxWarps * 32) {
        const int qr = i / pieces, ch = i - qr * pieces, qtl = qr / per;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (qtl < QT && t0 + qtl < p.num_tokens)
          v = *reinterpret_cast<const uint4*>(
              p.q + (static_cast<size_t>(t0 + qtl) * p.heads + g * per + (qr - qtl * per)) * (p.k_chunks * 64) + ch * 8);
        *reinterpret_cast<uint4*>(base_ptr + (ch >> 3) * kMpChunk + swz128(qr, ch & 7)) = v;
      }
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_q);
    }
    // slice entry of this row and key column c: distance (p0 + tl) - (tile key) - c
    const float* b_row = b_sm + min(head, per - 1) * p.bias_stride + min(tl, QT - 1) + (kMpKeys - 1) - hf * 64;
    float m_run = -INFINITY, l_run = 0.f;
    bool alive = true;
#pragma unroll 1
    for (int j = 0; j < n_tiles; ++j) {
      const int buf = j & 1;
      const float* bt = b_row + buf * per * p.bias_stride;
      if (alive) alive = mbar_wait(bar_bfull + 8 * buf, (j >> 1) & 1, p.err);
      if (alive) alive = mbar_wait(bar_sfull + 8 * buf, (j >> 1) & 1, p.err);
      tc_fence_after();
      float s[64];
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t raw[32];
        tmem_ld32(lane_addr + buf * kMpKeys + hf * 64 + half * 32, raw);
        tmem_ld_wait();
#pragma unroll
        for (int c = 0; c < 32; ++c) {
          const int cc = half * 32 + c;
          s[cc] = fmaf(__uint_as_float(raw[c]), kMpLog2e, -bt[-cc]);
          mx4[c & 3] = fmaxf(mx4[c & 3], s[cc]);
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) {
        mbar_arrive(bar_bempty + 8 * buf);
        if (!kAlias) mbar_arrive(bar_sempty + 8 * buf);  // this S accumulator may be overwritten
      }
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      float* mxb = mx_sm + buf * 2 * kMpRows;
      mxb[hf * kMpRows + r] = mx;
      mp_pair_barrier(quarter);
      const float m_new = fmaxf(m_run, fmaxf(mx, mxb[(hf ^ 1) * kMpRows + r]));
      const bool need = m_new - m_run > kMpRescaleLog2;  // true on the first tile a row sees (m_run = -inf)
      // O, and P's place, are free once the product of the tile before has finished
      if (j > 0 && alive) alive = mbar_wait(bar_odone, (j - 1) & 1, p.err);
      tc_fence_after();
      if (__any_sync(0xffffffffu, need)) {
        if (j > 0) {
          const float alpha = m_new == -INFINITY ? 1.f : mp_exp2(m_run - m_new);
          l_run *= alpha;
#pragma unroll
          for (int c0 = 0; c0 < DV / 2; c0 += 32) {
            uint32_t o[32];
            tmem_ld32(tmem_o + c0, o);
            tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < 32; ++c) o[c] = __float_as_uint(__uint_as_float(o[c]) * alpha);
            mp_tmem_st32(tmem_o + c0, o);
          }
        }
        m_run = m_new;
      }
      const float mb = m_run == -INFINITY ? 0.f : m_run;
      float sum4[4] = {0.f, 0.f, 0.f, 0.f};
      uint32_t pw[32];
#pragma unroll
      for (int c = 0; c < 32; ++c) {
        const float e0 = mp_exp2(s[2 * c] - mb), e1 = mp_exp2(s[2 * c + 1] - mb);
        sum4[c & 3] += e0 + e1;
        pw[c] = pack_bf16x2(e0, e1);
      }
      l_run += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
      mp_tmem_st32(lane_addr + (kAlias ? buf * kMpKeys : 448) + hf * 32, pw);
      mp_tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) {
        mbar_arrive(bar_pfull);
        if (kAlias) mbar_arrive(bar_sempty + 8 * buf);
      }
    }
    if (alive) alive = mbar_wait(bar_odone, (n_tiles - 1) & 1, p.err);
    tc_fence_after();
    l_sm[hf * kMpRows + r] = l_run;
    mp_pair_barrier(quarter);
    const float inv = p.out_scale / (l_run + l_sm[(hf ^ 1) * kMpRows + r]);
    __nv_bfloat16* orow = p.out + static_cast<size_t>(t0 + tl) * p.out_ld + static_cast<size_t>(g * per + head) * DV + hf * (DV / 2);
#pragma unroll
    for (int c0 = 0; c0 < DV / 2; c0 += 32) {
      uint32_t o[32];
      tmem_ld32(tmem_o + c0, o);
      tmem_ld_wait();
      if (real && alive) {
#pragma unroll
        for (int c = 0; c < 32; c += 8) {
          uint4 w;
          w.x = pack_bf16x2(__uint_as_float(o[c]) * inv, __uint_as_float(o[c + 1]) * inv);
          w.y = pack_bf16x2(__uint_as_float(o[c + 2]) * inv, __uint_as_float(o[c + 3]) * inv);
          w.z = pack_bf16x2(__uint_as_float(o[c + 4]) * inv, __uint_as_float(o[c + 5]) * inv);
          w.w = pack_bf16x2(__uint_as_float(o[c + 6]) * inv, __uint_as_float(o[c + 7]) * inv);
          *reinterpret_cast<uint4*>(orow + c0 + c) = w;
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
#endif
}

// Floats per head of a slice: a step of 32 / per (per a power of two up to 32) puts the 32 rows of a warp into 32 banks.
static int mixed_bias_stride(int per) {
  const int need = kMpKeys + kMpRows / per;
  int step = 1;
  while (step * per < 32) step <<= 1;
  int s = (need + 31) / 32 * 32 + step;
  if (s - 32 >= need) s -= 32;
  return s;
}

// Stages of the K ring that fit beside the queries, the values and the slices; below 2 the kernel is not used.
static int mixed_prefill_stages(int heads, int kv_heads, int key_dim, int value_dim, size_t* smem_out) {
  if (heads % kv_heads || heads / kv_heads > kMpRows || key_dim % 64 || value_dim % 64 || value_dim > 256) return 0;
  const int per = heads / kv_heads, chunks = kv_heads * key_dim / 64;
  const size_t fixed = 1024 + 256 + (4 + 2) * kMpRows * 4 + static_cast<size_t>(2) * per * mixed_bias_stride(per) * 4 +
                       static_cast<size_t>(chunks + value_dim / 64) * kMpChunk;
  const size_t room = 227 * 1024;
  if (fixed >= room) return 0;
  int stages = static_cast<int>((room - fixed) / kMpChunk);
  if (stages > kMpMaxStages) stages = kMpMaxStages;
  if (smem_out) *smem_out = fixed + static_cast<size_t>(stages) * kMpChunk;
  return stages;
}

template <int DV>
static int launch_mixed_prefill(const CUtensorMap& qm, const CUtensorMap& km, const CUtensorMap& vm, const MixedPrefillParams& p,
                                size_t smem, cudaStream_t st) {
  int rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&mixed_prefill_tc_kernel<DV>), 227 * 1024);
  if (rc) return rc;
  const int qt = kMpRows / (p.heads / p.kv_heads);
  B200_CUDA(launch_overlapped(mixed_prefill_tc_kernel<DV>, dim3((p.num_tokens + qt - 1) / qt, p.kv_heads), dim3(kMpThreads), smem, st,
                              qm, km, vm, p));
  return 0;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_mixed_attn_prefill_supported(int num_q_heads, int num_kv_heads, int key_dim, int value_dim) {
  if (num_q_heads <= 0 || num_kv_heads <= 0 || key_dim <= 0 || value_dim <= 0 || num_kv_heads > 65535) return 0;
  return mixed_prefill_stages(num_q_heads, num_kv_heads, key_dim, value_dim, nullptr) >= 2;
}

extern "C" int b200_mixed_attn_prefill(const void* q, const void* k_pool, const void* v_pool, const int32_t* block_table_row,
                                       const float* bias, int bias_ld, int window, void* out, int out_ld, float out_scale,
                                       void* status_word, int num_tokens, int first_position, int num_q_heads, int num_kv_heads,
                                       int key_dim, int value_dim, int page_size, int num_blocks, int max_pages_per_seq,
                                       void* stream) {
  B200_REQUIRE(q && k_pool && v_pool && block_table_row && bias && out, "mixed_attn_prefill: null pointer");
  B200_REQUIRE(num_tokens > 0 && first_position >= 0 && page_size == kMpPage && num_blocks > 0 && window > 0 &&
                   first_position + num_tokens <= static_cast<long long>(max_pages_per_seq) * page_size,
               "mixed_attn_prefill: %d tokens from %d, pages of %d, window %d", num_tokens, first_position, page_size, window);
  size_t smem = 0;
  const int stages = b200_mixed_attn_prefill_supported(num_q_heads, num_kv_heads, key_dim, value_dim)
                         ? mixed_prefill_stages(num_q_heads, num_kv_heads, key_dim, value_dim, &smem) : 0;
  B200_REQUIRE(stages >= 2, "mixed_attn_prefill: not built for %d query heads over %d, key size %d, value size %d", num_q_heads,
               num_kv_heads, key_dim, value_dim);
  const long long seen = first_position + num_tokens < window ? first_position + num_tokens : window;
  B200_REQUIRE(bias_ld >= seen && out_ld >= num_q_heads * value_dim && out_ld % 8 == 0,
               "mixed_attn_prefill: bias rows of %d, output rows of %d", bias_ld, out_ld);
  B200_REQUIRE(aligned16({q, k_pool, v_pool, out}), "mixed_attn_prefill: buffers must be 16-byte aligned");
  int rc = check_device(nullptr);
  if (rc) return rc;
  const int per = num_q_heads / num_kv_heads;
  MixedPrefillParams p{};
  p.table_row = block_table_row;
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.bias = bias;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.err = static_cast<int*>(status_word);
  p.bias_ld = bias_ld;
  p.window = window;
  p.out_ld = out_ld;
  p.out_scale = out_scale;
  p.num_tokens = num_tokens;
  p.first_pos = first_position;
  p.heads = num_q_heads;
  p.kv_heads = num_kv_heads;
  p.num_blocks = num_blocks;
  p.dk_chunks = key_dim / 64;
  p.k_chunks = num_kv_heads * p.dk_chunks;
  p.stages = stages;
  p.q_tma = per % 8 == 0 && 128 % per == 0;
  p.bias_stride = mixed_bias_stride(per);
  CUtensorMap qm, km, vm;
  const uint64_t rows = static_cast<uint64_t>(num_blocks) * num_kv_heads * kMpPage;
  rc = get_tensor_map_2d(k_pool, rows, key_dim, 2, kMpPage, 64, &km);
  if (rc) return rc;
  rc = get_tensor_map_2d(v_pool, rows, value_dim, 2, kMpPage, 64, &vm);
  if (rc) return rc;
  qm = km;
  if (p.q_tma) {
    rc = get_tensor_map_2d(q, static_cast<uint64_t>(num_tokens) * num_q_heads, static_cast<uint64_t>(p.k_chunks) * 64, 2, per, 64, &qm);
    if (rc) return rc;
  }
  cudaStream_t st = as_stream(stream);
  switch (value_dim) {
    case 64: return launch_mixed_prefill<64>(qm, km, vm, p, smem, st);
    case 128: return launch_mixed_prefill<128>(qm, km, vm, p, smem, st);
    case 192: return launch_mixed_prefill<192>(qm, km, vm, p, smem, st);
    default: return launch_mixed_prefill<256>(qm, km, vm, p, smem, st);
  }
}
