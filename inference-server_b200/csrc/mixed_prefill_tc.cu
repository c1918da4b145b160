// Attention with mixed heads (see mixed_attn.cu) for a chunk of prompt tokens of one sequence on the tcgen05 tensor cores:
// bf16, key size a multiple of 64 per kv head, value size 64, 128, 192 or 256, up to 128 query heads per kv head.
//
//   grid     (query tiles, kv heads).  A CTA owns 128 score rows: 128 / per consecutive positions x the `per` query heads of
//            its kv head, and walks the key tiles (128 keys = 8 pages) from the one that holds the first key its first row
//            sees to the one of its last position.
//   warp 0   K producer: a tile's keys of ALL kv heads, `nc` 64-wide columns (nc x 16 KiB) at a time, into a ring.  A box is 8 tokens
//            of nc columns; the 16 boxes of a tile lie one after the other, so groups of 8 keys are nc KiB apart and every column is
//            a K-major B operand as it lands.
//   warp 1   issuer (one elected lane): S(0), then S(j + 1) and O += P(j) V(j) for every tile j.  S = Q' K^T is 4 x tcgen05.mma
//            M128 N128 K16 per 64 columns; V is an MN-major B operand straight from its page layout.  While the softmax of
//            tile j runs, S(j + 1) is in the tensor pipe.
//   warp 2   the distance table (log2 units): per tile a bulk copy of the slice of B[h][.] that the tile's rows and keys meet.
//            It is +inf where a distance is negative (a later token) or outside the window, so the mask costs nothing.
//   warp 3   V producer: the values of the CTA's kv head, one tile at a time, a box per page.
//   warps 4-11  softmax: a thread owns a score row and 64 of the tile's 128 keys (TMEM lanes are bound to warp_id % 4; the two
//            warps with the same rows meet on a named barrier for the row maximum).  s = score * log2 e - B from the slice in
//            shared memory, lazy rescale of O as in paged_prefill_tc.cu, P = exp2(s - m) as bf16.
//
// The mixed queries meet the keys of all kv heads, so they are kv_heads times as wide as a head, and so is a tile of keys: what a
// CTA can have in flight decides its speed.  Two forms (QTMEM):
//   true   Q' is an A operand in TMEM (columns / 2 of it), beside O and one or two S accumulators; P goes through shared memory,
//          which is left to the ring.  Whenever those fit the 512 columns.  The CTA mixes the raw queries itself, on the tensor
//          cores: per kv head c, Q'_c = T_c q_c, where q_c holds the tile's raw queries of that head (rows position x head) and T_c
//          repeats the mixing matrix's block (the CTA's heads x the heads of c) along its diagonal, once per position.  q_c comes
//          through the ring, T_c is written into P's place, the product goes through the S accumulator into Q'.
//   false  Q', mixed already (b200_mix_heads), in shared memory; S0 columns 0-127, S1 128-255, O from 256 on, P in the last 64
//          columns; with value size 256, where none are left, P(j) lies over S(j), and the issuer waits for the product with P(j)
//          before it writes that S again.
// Every mbarrier wait is bounded; one that runs out records kErrDevWaitTimeout, and the thread stops waiting but keeps the loop
// structure (the named barriers between partner warps are still met), so the kernel ends.

#include "glue.cuh"

namespace b200 {

constexpr int kMpPage = 16;
constexpr int kMpRows = 128, kMpKeys = 128;
constexpr int kMpChunk = 128 * 128;  // 128 rows x 64 bf16
constexpr int kMpSoftmaxWarps = 8;
constexpr int kMpThreads = (4 + kMpSoftmaxWarps) * 32;
constexpr int kMpMaxStages = 12;
constexpr int kMpBarBytes = 384;  // barriers, tmem base
constexpr float kMpRescaleLog2 = 8.f;
constexpr float kMpLog2e = 1.4426950408889634f;

struct MixedPrefillParams {
  const int* table_row;
  const __nv_bfloat16* q;  // !QTMEM: [tokens, heads, k_chunks * 64]
  const __nv_bfloat16* talk;  // QTMEM: the mixing matrix [heads, heads]
  const float* bias;       // [heads, bias_ld]
  __nv_bfloat16* out;      // [tokens, out_ld]
  int* err;
  int bias_ld, window, out_ld;
  float out_scale, score_scale;  // score_scale: log2 e, with the scores' own factor where that is not in q
  int num_tokens, first_pos, heads, kv_heads, num_blocks;
  int k_chunks;            // 64-wide pieces of a mixed query (all kv heads)
  int dk_chunks;           // of one kv head's keys
  int nc, stages, s_bufs;  // 64-wide pieces of a stage
  int bias_stride;         // floats per head of a slice
};

__host__ __device__ constexpr uint32_t mp_idesc(uint32_t n, uint32_t b_mn) {
  return (1u << 4) | (1u << 7) | (1u << 10) | (b_mn << 16) | ((n >> 3) << 17) | ((128u >> 4) << 24);
}
// Issued by a converged warp: one elected lane sends the instruction, and the descriptors, the same in all lanes, can stay in
// uniform registers (a branch on the lane number around the loop costs more than the instructions themselves).
__device__ __forceinline__ void mp_mma_ss(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p, e;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "@e tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}" ::"r"(d), "l"(a), "l"(b), "r"(idesc), "r"(acc)
      : "memory");
}
// A from TMEM: lane = row, a 32-bit column = two neighbouring K elements.
__device__ __forceinline__ void mp_mma_ts(uint32_t d, uint32_t a, uint64_t b, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p, e;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "@e tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}" ::"r"(d), "r"(a), "l"(b), "r"(idesc), "r"(acc)
      : "memory");
}
__device__ __forceinline__ void mp_commit(uint32_t bar) {
  asm volatile(
      "{\n\t.reg .pred e;\n\t"
      "elect.sync _|e, 0xffffffff;\n\t"
      "@e tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}" ::"r"(bar)
      : "memory");
}
// A wait of a whole warp, true if it has not run out for any lane.
__device__ __forceinline__ bool mp_wait_all(uint32_t bar, uint32_t parity, int* err) {
  return __all_sync(0xffffffffu, mbar_wait(bar, parity, err));
}
// Operand descriptors, 128-byte swizzle.  MN-major (16 K rows of it): the next 8 K rows are 1024 bytes, the next 64 columns 2048
// bytes further.  K-major: groups of 8 rows are `sbo` bytes apart.
__device__ __forceinline__ uint64_t mp_desc_mn(uint32_t addr) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((addr & 0x3FFFFu) >> 4);
  d |= static_cast<uint64_t>(2048 >> 4) << 16;
  d |= static_cast<uint64_t>(1024 >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
__device__ __forceinline__ uint64_t mp_desc_k(uint32_t addr, uint32_t sbo) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((addr & 0x3FFFFu) >> 4);
  d |= static_cast<uint64_t>(1) << 16;
  d |= static_cast<uint64_t>(sbo >> 4) << 32;
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
__device__ __forceinline__ void mp_pair_barrier(int quarter) {
  switch (quarter) {
    case 0: asm volatile("bar.sync 1, 64;" ::: "memory"); break;
    case 1: asm volatile("bar.sync 2, 64;" ::: "memory"); break;
    case 2: asm volatile("bar.sync 3, 64;" ::: "memory"); break;
    default: asm volatile("bar.sync 4, 64;" ::: "memory"); break;
  }
}

template <int DV, bool QTMEM>
__global__ void __launch_bounds__(kMpThreads, 1)
mixed_prefill_tc_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map,
                        const __grid_constant__ CUtensorMap v_map, const MixedPrefillParams p) {
#ifdef B200_DEVICE_OK
  constexpr int kVChunks = DV / 64;
  constexpr bool kAlias = !QTMEM && DV > 192;  // P over S
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
  // Q' or P (two halves of 64 keys), V, the ring of keys
  const int first_chunks = QTMEM ? 2 : p.k_chunks;
  const uint32_t q_sm = base, v_sm = q_sm + first_chunks * kMpChunk, k_sm = v_sm + kVChunks * kMpChunk;
  const uint32_t stage_bytes = static_cast<uint32_t>(p.nc) * kMpChunk;
  uint8_t* extra = base_ptr + (first_chunks + kVChunks + p.stages * p.nc) * kMpChunk;
  const uint32_t bars = k_sm + p.stages * stage_bytes;
  const uint32_t bar_q = bars, bar_vfull = bars + 8, bar_vempty = bars + 16;
  const uint32_t bar_sfull = bars + 24, bar_sempty = bars + 40;  // [2] each
  const uint32_t bar_pfull = bars + 56, bar_odone = bars + 64;
  const uint32_t bar_bfull = bars + 72, bar_bempty = bars + 88;  // [2] each: slice of the distance table
  const uint32_t bar_a = bars + 104, bar_rfull = bars + 112, bar_rempty = bars + 120;  // mixing: T_c written; a round's product
  const uint32_t bar_kfull = bars + 128, bar_kempty = bar_kfull + 8 * kMpMaxStages;
  uint32_t* tmem_base_sm = reinterpret_cast<uint32_t*>(extra + kMpBarBytes - 16);
  float* mx_sm = reinterpret_cast<float*>(extra + kMpBarBytes);  // [2 tiles][2 halves][128 rows]
  float* l_sm = mx_sm + 2 * 2 * kMpRows;                 // [2 halves][128 rows]
  float* b_sm = l_sm + 2 * kMpRows;                      // [2][per][bias_stride]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per = p.heads / p.kv_heads, QT = kMpRows / per;
  if (threadIdx.x == 32) {
    if (QTMEM) tma_prefetch_desc(&q_map);
    tma_prefetch_desc(&k_map);
    tma_prefetch_desc(&v_map);
  }
  if (threadIdx.x == 0) {
    mbar_init(bar_q, kMpSoftmaxWarps);
    mbar_init(bar_a, kMpSoftmaxWarps);
    mbar_init(bar_rfull, 1);
    mbar_init(bar_rempty, kMpSoftmaxWarps);
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
  if (QTMEM && QT * per < kMpRows) {  // raw queries fill QT * per rows of a piece; the rest meets zero columns of T_c and must be finite
    const int tail = (kMpRows - QT * per) * 8;  // 16-byte pieces
    for (int i = threadIdx.x; i < p.stages * p.nc * tail; i += kMpThreads) {
      const int c = i / tail;
      *reinterpret_cast<uint4*>(base_ptr + (first_chunks + kVChunks + c) * kMpChunk + QT * per * 128 + (i - c * tail) * 16) =
          make_uint4(0u, 0u, 0u, 0u);
    }
    fence_proxy_async();
  }
  if (warp == 1) tmem_alloc(smem_u32(tmem_base_sm), 512);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_base_sm;
  // columns: QTMEM  O, Q', S buffers;  else  S0, S1, O, P
  const uint32_t o_col = QTMEM ? 0u : 256u, q_col = DV, s_col = QTMEM ? DV + p.k_chunks * 32u : 0u;
  const int s_bufs = QTMEM ? p.s_bufs : 2;
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
    bool alive = true;
    uint32_t slot = 0, kphase = 1;
    if (QTMEM && warp == 0) {  // the raw queries of all heads, a box per 64-wide piece: rows position x head
#pragma unroll 1
      for (int s0 = 0; s0 < p.k_chunks && alive; s0 += p.nc) {
        alive = mp_wait_all(bar_kempty + 8 * slot, kphase, p.err);
        if (!alive) break;
        if (lane == 0) mbar_arrive_expect_tx(bar_kfull + 8 * slot, static_cast<uint32_t>(p.nc * QT * per) * 128u);
        __syncwarp();
        if (lane < p.nc) {
          const int c = (s0 + lane) / p.dk_chunks;
          tma_load_3d(k_sm + slot * stage_bytes + lane * kMpChunk, &q_map, bar_kfull + 8 * slot, (s0 + lane - c * p.dk_chunks) * 64,
                      c * per, t0);
        }
        if (++slot == static_cast<uint32_t>(p.stages)) {
          slot = 0;
          kphase ^= 1;
        }
      }
    }
#pragma unroll 1
    for (int j = 0; j < n_tiles && alive; ++j) {
      // pages past the last position stand in for by it: their keys are masked, their values meet weights of 0
      int page = 0;
      if (lane < 8) {
        page = __ldg(p.table_row + min((kt0 + j) * 8 + lane, last_page));
        if (page < 0 || page >= p.num_blocks) {
          set_error(p.err, kErrDevBadBlockId);
          page = 0;
        }
      }
      if (warp == 0) {
        const int my_page = __shfl_sync(0xffffffffu, page, (lane >> 1) & 7);  // lanes 0-15: half a page each
#pragma unroll 1
        for (int s0 = 0; s0 < p.k_chunks; s0 += p.nc) {
          alive = mp_wait_all(bar_kempty + 8 * slot, kphase, p.err);
          if (!alive) break;
          if (lane == 0) mbar_arrive_expect_tx(bar_kfull + 8 * slot, stage_bytes);
          __syncwarp();
          if (lane < 16)
            tma_load_3d(k_sm + slot * stage_bytes + lane * (p.nc * 1024), &k_map, bar_kfull + 8 * slot, 0, (lane & 1) * 8,
                        my_page * p.k_chunks + s0);
          if (++slot == static_cast<uint32_t>(p.stages)) {
            slot = 0;
            kphase ^= 1;
          }
        }
      } else {
        alive = mp_wait_all(bar_vempty, (j & 1) ^ 1, p.err);
        if (!alive) break;
        if (lane == 0) mbar_arrive_expect_tx(bar_vfull, kVChunks * kMpChunk);
        __syncwarp();
        if (lane < 8)
          tma_load_2d(v_sm + lane * (kVChunks * 2048), &v_map, bar_vfull, 0, (page * p.kv_heads + g) * kVChunks * kMpPage);
      }
    }
  } else if (warp == 1) {
    // ---------------------------------------------------------------- issuer ------
    constexpr uint32_t idesc_s = mp_idesc(kMpKeys, 0), idesc_o = mp_idesc(DV, 1);
    const uint32_t tmem_o = tmem_base + o_col;
    uint32_t slot = 0, kphase = 0;
    const uint64_t q_desc = umma_desc_k128(q_sm), k_desc = mp_desc_k(k_sm, p.nc * 1024), v_desc = mp_desc_mn(v_sm);
    bool alive = true;
    if (QTMEM) {  // mix the queries: rounds of up to two 64-wide pieces of a kv head through the first S accumulator
      constexpr uint32_t idesc_mix = mp_idesc(64, 1);
      int round = 0, c = 0, cc = 0;
#pragma unroll 1
      for (int s0 = 0; s0 < p.k_chunks && alive; s0 += p.nc) {
        alive = mp_wait_all(bar_kfull + 8 * slot, kphase, p.err);
#pragma unroll 1
        for (int i = 0; i < p.nc && alive; ++i) {
          if (cc == 0) alive = mp_wait_all(bar_a, c & 1, p.err);
          if ((cc & 1) == 0 && round > 0 && alive) alive = mp_wait_all(bar_rempty, (round - 1) & 1, p.err);
          if (!alive) break;
          tc_fence_after();
          const uint64_t b = mp_desc_mn(k_sm + slot * stage_bytes + i * kMpChunk);
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            mp_mma_ss(tmem_base + s_col + (cc & 1) * 64, q_desc + (kk >> 2) * (kMpChunk >> 4) + 2 * (kk & 3), b + kk * (2048 >> 4),
                      idesc_mix, kk > 0 ? 1u : 0u);
          const bool last = cc + 1 == p.dk_chunks;
          if ((cc & 1) != 0 || last) {
            mp_commit(bar_rfull);
            ++round;
          }
          cc = last ? 0 : cc + 1;
          c += last ? 1 : 0;
        }
        mp_commit(bar_kempty + 8 * slot);
        if (++slot == static_cast<uint32_t>(p.stages)) {
          slot = 0;
          kphase ^= 1;
        }
      }
      if (alive) alive = mp_wait_all(bar_rempty, (round - 1) & 1, p.err);  // the last of Q' is in place
    } else {
      alive = mp_wait_all(bar_q, 0, p.err);
    }
    auto scores = [&](int t) {
      const int sb = s_bufs == 2 ? t & 1 : 0;
      const uint32_t ph = (s_bufs == 2 ? t >> 1 : t) & 1, s_acc = tmem_base + s_col + sb * kMpKeys;
      if (alive) alive = mp_wait_all(bar_sempty + 8 * sb, ph ^ 1, p.err);
      if (kAlias && t >= 2 && alive) alive = mp_wait_all(bar_odone, (t - 2) & 1, p.err);  // P(t - 2) lies there
#pragma unroll 1
      for (int c = 0; c < p.k_chunks && alive; c += p.nc) {
        alive = mp_wait_all(bar_kfull + 8 * slot, kphase, p.err);
        if (!alive) break;
        tc_fence_after();
#pragma unroll 1
        for (int i = 0; i < p.nc; ++i) {
          const uint64_t a0 = q_desc + static_cast<uint32_t>(c + i) * (kMpChunk >> 4);
          const uint64_t b0 = k_desc + ((slot * stage_bytes + i * 1024u) >> 4);
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            if (QTMEM) mp_mma_ts(s_acc, tmem_base + q_col + (c + i) * 32 + k * 8, b0 + 2 * k, idesc_s, (c + i + k) > 0 ? 1u : 0u);
            else mp_mma_ss(s_acc, a0 + 2 * k, b0 + 2 * k, idesc_s, (c + i + k) > 0 ? 1u : 0u);
          }
        }
        mp_commit(bar_kempty + 8 * slot);
        if (++slot == static_cast<uint32_t>(p.stages)) {
          slot = 0;
          kphase ^= 1;
        }
      }
      if (alive) mp_commit(bar_sfull + 8 * sb);
    };
    scores(0);
#pragma unroll 1
    for (int j = 0; j < n_tiles && alive; ++j) {
      if (j + 1 < n_tiles) scores(j + 1);
      if (alive) alive = mp_wait_all(bar_vfull, j & 1, p.err);
      if (alive) alive = mp_wait_all(bar_pfull, j & 1, p.err);
      if (!alive) break;
      tc_fence_after();
      const uint32_t pa = tmem_base + (kAlias ? static_cast<uint32_t>((j & 1) * kMpKeys) : 448u);
#pragma unroll
      for (int kk = 0; kk < 8; ++kk) {
        const uint64_t b = v_desc + kk * ((kVChunks * 2048) >> 4);  // a page
        if (QTMEM) mp_mma_ss(tmem_o, q_desc + (kk >> 2) * (kMpChunk >> 4) + 2 * (kk & 3), b, idesc_o, (j > 0 || kk > 0) ? 1u : 0u);
        else mp_mma_ts(tmem_o, pa + kk * 8, b, idesc_o, (j > 0 || kk > 0) ? 1u : 0u);
      }
      mp_commit(bar_odone);
      mp_commit(bar_vempty);
    }
  } else if (warp == 2) {
    // ------------------------------------------- slices of the distance table ------
    // entry x of a head: distance p0 - (first key of the tile) - 127 + x, after up to 3 entries that make the copy's start a
    // multiple of 16 bytes
    bool alive = true;
    const int span = kMpKeys + QT - 1;
#pragma unroll 1
    for (int j = 0; j < n_tiles && alive; ++j) {
      alive = mp_wait_all(bar_bempty + 8 * (j & 1), ((j >> 1) & 1) ^ 1, p.err);
      if (!alive) break;
      const int at = kDistPad + p0 - (kt0 + j) * kMpKeys - (kMpKeys - 1);
      const uint32_t bytes = static_cast<uint32_t>(((at & 3) + span + 3) & ~3) * 4u;
      if (lane == 0) mbar_arrive_expect_tx(bar_bfull + 8 * (j & 1), bytes * per);
      __syncwarp();
      const uint32_t dst = smem_u32(b_sm) + static_cast<uint32_t>((j & 1) * per * p.bias_stride) * 4u;
      for (int hh = lane; hh < per; hh += 32)
        bulk_load(dst + static_cast<uint32_t>(hh * p.bias_stride) * 4u,
                  p.bias + static_cast<size_t>(g * per + hh) * p.bias_ld + (at & ~3), bytes, bar_bfull + 8 * (j & 1));
    }
  } else {
    // --------------------------------------------------------------- softmax ------
    const int sw = warp - 4, hf = sw >> 2, quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(quarter * 32) << 16);
    const uint32_t tmem_o = lane_addr + o_col + hf * (DV / 2);
    const int tl = r / per, head = r - tl * per;
    const bool real = tl < QT && t0 + tl < p.num_tokens;
    bool alive = true;
    if (QTMEM) {
#pragma unroll
      for (int i = 0; i < 8; ++i)
        *reinterpret_cast<uint4*>(base_ptr + ((sw * 32 + lane) * 8 + i) * 16) = make_uint4(0u, 0u, 0u, 0u);
      asm volatile("bar.sync 5, %0;" ::"n"(kMpSoftmaxWarps * 32) : "memory");
      int round = 0;
      const __nv_bfloat16* t = p.talk + static_cast<size_t>(g * per + head) * p.heads;
      __nv_bfloat16 row[8];  // the row's first factors for the next kv head, asked for ahead
#pragma unroll
      for (int x = 0; x < 8; ++x)
        if (x < per) row[x] = t[x];
#pragma unroll 1
      for (int c = 0; c < p.kv_heads; ++c) {
        if (hf == 0 && tl < QT) {  // this row of T_c: the CTA's head against the heads of c, at the row's position
          const auto put = [&](int x, __nv_bfloat16 v) {
            const int col = tl * per + x;
            *reinterpret_cast<__nv_bfloat16*>(base_ptr + (col >> 6) * kMpChunk + swz128(r, (col & 63) >> 3) + (col & 7) * 2) = v;
          };
#pragma unroll
          for (int x = 0; x < 8; ++x)
            if (x < per) put(x, row[x]);
          for (int x = 8; x < per; ++x) put(x, t[c * per + x]);
        }
        if (c + 1 < p.kv_heads)
#pragma unroll
          for (int x = 0; x < 8; ++x)
            if (x < per) row[x] = t[(c + 1) * per + x];
        fence_proxy_async();
        __syncwarp();
        if (lane == 0) mbar_arrive(bar_a);
#pragma unroll 1
        for (int cc = 0; cc < p.dk_chunks; cc += 2, ++round) {
          if (alive) alive = mbar_wait(bar_rfull, round & 1, p.err);
          tc_fence_after();
          if (cc + hf < p.dk_chunks) {
            uint32_t v[32], w[32];
#pragma unroll
            for (int half = 0; half < 2; ++half) {
              tmem_ld32(lane_addr + s_col + hf * 64 + half * 32, v);
              tmem_ld_wait();
#pragma unroll
              for (int e = 0; e < 16; ++e) w[half * 16 + e] = pack_bf16x2(__uint_as_float(v[2 * e]), __uint_as_float(v[2 * e + 1]));
            }
            mp_tmem_st32(lane_addr + q_col + (c * p.dk_chunks + cc + hf) * 32, w);
            mp_tmem_st_wait();
          }
          tc_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(bar_rempty);
        }
      }
    } else {  // the mixed queries, zero rows past the tile's last position; neighbouring threads take neighbouring 16-byte pieces
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
    const float* b_row = b_sm + head * p.bias_stride + min(tl, QT - 1) + (kMpKeys - 1) - hf * 64 +
                         ((kDistPad + p0 - (kMpKeys - 1)) & 3);  // a tile's first key is a multiple of 128
    float m_run = -INFINITY, l_run = 0.f;
#pragma unroll 1
    for (int j = 0; j < n_tiles; ++j) {
      const int buf = j & 1, sb = s_bufs == 2 ? buf : 0;
      const float* bt = b_row + buf * per * p.bias_stride;
      if (alive) alive = mbar_wait(bar_bfull + 8 * buf, (j >> 1) & 1, p.err);
      if (alive) alive = mbar_wait(bar_sfull + 8 * sb, (s_bufs == 2 ? j >> 1 : j) & 1, p.err);
      tc_fence_after();
      float s[64];
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t raw[32];
        tmem_ld32(lane_addr + s_col + sb * kMpKeys + hf * 64 + half * 32, raw);
        tmem_ld_wait();
#pragma unroll
        for (int c = 0; c < 32; ++c) {
          const int cc = half * 32 + c;
          s[cc] = fmaf(__uint_as_float(raw[c]), p.score_scale, -bt[-cc]);
          mx4[c & 3] = fmaxf(mx4[c & 3], s[cc]);
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) {
        mbar_arrive(bar_bempty + 8 * buf);
        if (!kAlias) mbar_arrive(bar_sempty + 8 * sb);  // this S accumulator may be overwritten
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
          const float alpha = m_new == -INFINITY ? 1.f : fast_ex2(m_run - m_new);
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
        const float e0 = fast_ex2(s[2 * c] - mb), e1 = fast_ex2(s[2 * c + 1] - mb);
        sum4[c & 3] += e0 + e1;
        pw[c] = pack_bf16x2(e0, e1);
      }
      l_run += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
      if (QTMEM) {
        uint8_t* p_half = base_ptr + hf * kMpChunk;
#pragma unroll
        for (int ch = 0; ch < 8; ++ch)
          *reinterpret_cast<uint4*>(p_half + swz128(r, ch)) = make_uint4(pw[4 * ch], pw[4 * ch + 1], pw[4 * ch + 2], pw[4 * ch + 3]);
        mp_tmem_st_wait();    // a rescaled O
        fence_proxy_async();  // the tensor core reads P through the async proxy
      } else {
        mp_tmem_st32(lane_addr + (kAlias ? buf * kMpKeys : 448) + hf * 32, pw);
        mp_tmem_st_wait();
      }
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

// Floats per head of a slice (rows of 16 bytes): a step of 32 / per (per a power of two up to 8) puts the 32 rows of a warp into
// 32 banks.
static int mixed_bias_stride(int per) {
  const int need = kMpKeys + kMpRows / per + 6;
  int step = 4;
  while (step * per < 32) step <<= 1;
  int s = (need + 31) / 32 * 32 + step;
  if (s - 32 >= need) s -= 32;
  return s;
}

// How the kernel runs for a shape: stages of the ring (below 2: not built for it), whether Q' lies in TMEM, S accumulators.
struct MixedPrefillPlan {
  int nc, stages, q_tmem, s_bufs;
  size_t smem;
};
static MixedPrefillPlan mixed_prefill_plan(int heads, int kv_heads, int key_dim, int value_dim) {
  MixedPrefillPlan pl{1, 0, 0, 2, 0};
  if (heads % kv_heads || heads / kv_heads > kMpRows || key_dim % 64 || value_dim % 64 || value_dim > 256) return pl;
  const int per = heads / kv_heads, chunks = kv_heads * key_dim / 64, columns = value_dim + chunks * 32;
  if (columns + kMpKeys <= 512) {
    pl.q_tmem = 1;
    pl.s_bufs = columns + 2 * kMpKeys <= 512 ? 2 : 1;
  }
  const size_t fixed = 1024 + kMpBarBytes + (4 + 2) * kMpRows * 4 + static_cast<size_t>(2) * per * mixed_bias_stride(per) * 4 +
                       static_cast<size_t>((pl.q_tmem ? 2 : chunks) + value_dim / 64) * kMpChunk;
  const size_t room = 227 * 1024;
  if (fixed >= room) return pl;
  // stages as large as leaves two of them: larger boxes cost the copy engine less
  for (int nc = 4; nc >= 1; --nc) {
    if (chunks % nc) continue;
    pl.nc = nc;
    pl.stages = static_cast<int>((room - fixed) / (static_cast<size_t>(nc) * kMpChunk));
    if (pl.stages >= 2) break;
  }
  if (pl.stages > kMpMaxStages) pl.stages = kMpMaxStages;
  pl.smem = fixed + static_cast<size_t>(pl.stages) * pl.nc * kMpChunk;
  return pl;
}

template <int DV, bool QTMEM>
static int launch_mixed_prefill(const CUtensorMap& qm, const CUtensorMap& km, const CUtensorMap& vm, const MixedPrefillParams& p, size_t smem, cudaStream_t st) {
  int rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&mixed_prefill_tc_kernel<DV, QTMEM>), 227 * 1024);
  if (rc) return rc;
  const int qt = kMpRows / (p.heads / p.kv_heads);
  B200_CUDA(launch_overlapped(mixed_prefill_tc_kernel<DV, QTMEM>, dim3((p.num_tokens + qt - 1) / qt, p.kv_heads), dim3(kMpThreads),
                              smem, st, qm, km, vm, p));
  return 0;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_mixed_attn_prefill_supported(int num_q_heads, int num_kv_heads, int key_dim, int value_dim) {
  if (num_q_heads <= 0 || num_kv_heads <= 0 || key_dim <= 0 || value_dim <= 0 || num_kv_heads > 65535) return 0;
  const MixedPrefillPlan plan = mixed_prefill_plan(num_q_heads, num_kv_heads, key_dim, value_dim);
  return plan.stages < 2 ? 0 : plan.q_tmem ? 2 : 1;
}

extern "C" int b200_mixed_attn_prefill(const void* q, const void* talk, float scale, const void* k_pool, const void* v_pool, const int32_t* block_table_row,
                                       const float* bias, int bias_ld, int window, void* out, int out_ld, float out_scale,
                                       void* status_word, int num_tokens, int first_position, int num_q_heads, int num_kv_heads,
                                       int key_dim, int value_dim, int page_size, int num_blocks, int max_pages_per_seq,
                                       void* stream) {
  B200_REQUIRE(q && k_pool && v_pool && block_table_row && bias && out, "mixed_attn_prefill: null pointer");
  B200_REQUIRE(num_tokens > 0 && first_position >= 0 && page_size == kMpPage && num_blocks > 0 && window > 0 &&
                   first_position + num_tokens <= static_cast<long long>(max_pages_per_seq) * page_size,
               "mixed_attn_prefill: %d tokens from %d, pages of %d, window %d", num_tokens, first_position, page_size, window);
  B200_REQUIRE(b200_mixed_attn_prefill_supported(num_q_heads, num_kv_heads, key_dim, value_dim), "mixed_attn_prefill: not built for %d query heads over %d, key size %d, value size %d", num_q_heads,
               num_kv_heads, key_dim, value_dim);
  const long long seen = first_position + num_tokens < window ? first_position + num_tokens : window;
  B200_REQUIRE(bias_ld >= kDistPad + seen + kDistTail && bias_ld % 4 == 0 && out_ld >= num_q_heads * value_dim && out_ld % 8 == 0,
               "mixed_attn_prefill: bias rows of %d, output rows of %d", bias_ld, out_ld);
  B200_REQUIRE(aligned16({q, k_pool, v_pool, out, bias}), "mixed_attn_prefill: buffers must be 16-byte aligned");
  int rc = check_device(nullptr);
  if (rc) return rc;
  const int per = num_q_heads / num_kv_heads;
  const MixedPrefillPlan plan = mixed_prefill_plan(num_q_heads, num_kv_heads, key_dim, value_dim);
  B200_REQUIRE(!plan.q_tmem || (talk && num_q_heads / num_kv_heads <= 256), "mixed_attn_prefill: raw queries need the mixing matrix");
  MixedPrefillParams p{};
  p.talk = static_cast<const __nv_bfloat16*>(talk);
  p.score_scale = (plan.q_tmem ? scale : 1.f) * kMpLog2e;
  p.nc = plan.nc;
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
  p.stages = plan.stages;
  p.s_bufs = plan.s_bufs;
  p.bias_stride = mixed_bias_stride(per);
  CUtensorMap qm, km, vm;
  rc = get_tensor_map_3d(k_pool, static_cast<uint64_t>(num_blocks) * p.k_chunks, kMpPage, 64, 2, p.nc, 8, 64, &km);
  if (rc) return rc;
  const int v_rows = value_dim / 64 * kMpPage;  // of a kv head and page
  rc = get_tensor_map_2d(v_pool, static_cast<uint64_t>(num_blocks) * num_kv_heads * v_rows, 64, 2, v_rows, 64, &vm);
  if (rc) return rc;
  qm = km;
  if (plan.q_tmem) {
    rc = get_tensor_map_3d(q, num_tokens, num_q_heads, key_dim, 2, kMpRows / per, per, 64, &qm);
    if (rc) return rc;
  }
  cudaStream_t st = as_stream(stream);
#define B200_MIXED_PREFILL(DV)                                                             \
  return plan.q_tmem ? launch_mixed_prefill<DV, true>(qm, km, vm, p, plan.smem, st)            \
                     : launch_mixed_prefill<DV, false>(qm, km, vm, p, plan.smem, st)
  switch (value_dim) {
    case 64: B200_MIXED_PREFILL(64);
    case 128: B200_MIXED_PREFILL(128);
    case 192: B200_MIXED_PREFILL(192);
    default: B200_MIXED_PREFILL(256);
  }
#undef B200_MIXED_PREFILL
}
