// The recurrences of state_scan.cu for a chunk of prompt tokens of one sequence, 64 tokens at a time on the tensor cores
// (mma.sync), bf16 activations, dim and vdim multiples of 16, dim at most 128.
//
// With G_t the product of the block's decays up to token t and S the state before the block (rows of q, k are raw; iq_t, ik_t
// are the factors that make them unit vectors, q's scale included, or 1):
//     P[t, s] = iq_t ik_s G_t / G_s (q_t . k_s),  s <= t            A[t, s] = beta_t ik_t ik_s G_t / G_s (k_t . k_s),  s < t
//     U = (I + A)^-1 diag(beta) (V - diag(G ik) K S)    (gated delta rule; otherwise U = V)
//     O = diag(G iq) Q S + P U                           S' = G_64 S + K^T diag(G_64 / G ik) U
// The prepare kernel makes P and T = (I + A)^-1 for all blocks and heads side by side; the block kernel walks the blocks in
// order, a CTA per head and 16 columns of the state, which stay in registers as accumulators.
//
// fp32 where the recurrence is: q, k and v enter as the bf16 numbers they are, all factors are applied to fp32 values, and every
// other operand of a product - S, U, P, T and the residuals - is split into the bf16 number next to it and the bf16 number next
// to what is left (16 bits of mantissa), whose products are summed in fp32.

#include "glue.cuh"

namespace b200 {

constexpr int kBlk = 64;             // tokens of a block
constexpr int kChunkThreads = 128;
constexpr int kSmLd = 24;            // pitch (bf16) of 16-column operands in shared memory: ldmatrix without conflicts
constexpr int kFragsPerBlock = 4 * 4 * 2 * 32;  // uint4: row tile, k step, high / low part, lane
constexpr int kFactors = 4;          // G iq, G ik, beta, G_64 / G ik

struct ChunkParams {
  const __nv_bfloat16* act;
  int ld, q_off, k_off, v_off;
  const float* ba;
  const float* a_log;
  const float* dt_bias;
  const float* decay;
  float* state;
  const int* slots;
  const int* positions;
  float* o;
  uint4* p_frags;    // [blocks, heads, kFragsPerBlock]
  uint4* t_frags;    // the same, gated delta rule
  float* factors;    // [blocks, heads, kFactors, 64], then [blocks, heads]: G_64
  int* err;
  int rows, blocks, heads, qk_heads, dim, vdim, num_slots;
  float q_scale;
};

__device__ __forceinline__ float chunk_log_decay(float a_log, float a, float dt_bias) {
  const float z = a + dt_bias;
  return -expf(a_log) * (z > 20.f ? z : log1pf(expf(z)));
}
// Two fp32 numbers as packed bf16 and what the rounding left.
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16x2(x - f.x, y - f.y);
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool have) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(have ? 16 : 0) : "memory");
}

// Room for the two tiles of the prepare kernel.
__host__ __device__ __forceinline__ int prep_k_bytes(int dim) {
  const int t = kBlk * (dim + 8) * 2;
  return t > 32 * 68 * 4 ? t : 32 * 68 * 4;
}
__host__ __device__ __forceinline__ int prep_q_bytes(int dim, bool delta) {
  const int t = kBlk * (dim + 8) * 2;
  return !delta || t > kBlk * 68 * 4 ? t : kBlk * 68 * 4;
}

// 64-row tiles of k and q into shared memory (k, then q `tile_bytes` further), rows of dim + 8, zero rows past the last token.  A
// thread keeps its 16-byte column; row and column are worked out once.
struct TileLoader {
  uint32_t dst;
  int row, step, col, ld;
  __device__ __forceinline__ TileLoader(int dim, int ld_, int t, int threads) {
    const int pieces = dim / 8;
    step = threads / pieces;
    row = t / pieces;
    col = (t - row * pieces) * 8;
    if (row >= step) row = kBlk;  // left over
    ld = ld_;
    dst = (row * (dim + 8) + col) * 2;
  }
  __device__ __forceinline__ void load(uint32_t sm, int tile_bytes, const __nv_bfloat16* k, const __nv_bfloat16* q, int cnt, int ldk) const {
    uint32_t d = sm + dst;
    const __nv_bfloat16* kp = k + static_cast<size_t>(row) * ld + col;
    const __nv_bfloat16* qp = q + static_cast<size_t>(row) * ld + col;
    const size_t hop = static_cast<size_t>(step) * ld;
    for (int r = row; r < kBlk; r += step) {
      const bool have = r < cnt;
      cp_async16(d, have ? kp : k, have);
      cp_async16(d + tile_bytes, have ? qp : q, have);
      d += step * ldk * 2;
      kp += hop;
      qp += hop;
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
};

// C[r][c] (+)= sign * sum over k < n of a[r][k] b[k][c] for an n x n tile (n 16 or 32) of fp32 rows of 68; a thread takes four
// columns of one row.  `threads` of them, numbered from 0.
template <int N>
__device__ __forceinline__ void small_product(const float* a, const float* b, float* c, float sign, int t, int threads) {
  for (int i = t; i < N * N / 4; i += threads) {
    const int r = i / (N / 4), c4 = (i - r * (N / 4)) * 4;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k < N; k += 4) {
      const float4 x = *reinterpret_cast<const float4*>(a + r * 68 + k);
      const float xs[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float4 y = *reinterpret_cast<const float4*>(b + (k + e) * 68 + c4);
        acc.x = fmaf(xs[e], y.x, acc.x);
        acc.y = fmaf(xs[e], y.y, acc.y);
        acc.z = fmaf(xs[e], y.z, acc.z);
        acc.w = fmaf(xs[e], y.w, acc.w);
      }
    }
    *reinterpret_cast<float4*>(c + r * 68 + c4) = make_float4(sign * acc.x, sign * acc.y, sign * acc.z, sign * acc.w);
  }
}

template <bool DELTA>
__global__ void __launch_bounds__(kChunkThreads)
chunk_prepare_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) uint8_t cp_sm[];
  __shared__ float L[kBlk], ikv[kBlk], iqv[kBlk], bt[kBlk];
  grid_dep_wait();
  grid_dep_launch();
  const int blk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, tq = lane & 3, lj = lane >> 3, lr = lane & 7;
  const int t0 = blk * kBlk, cnt = min(kBlk, p.rows - t0);
  const int qh = h / (p.heads / p.qk_heads), ldk = p.dim + 8;
  // k (later a scratch tile), q (later the inverse), A: fp32 tiles have rows of 68
  const int k_room = prep_k_bytes(p.dim), q_room = prep_q_bytes(p.dim, DELTA);
  const uint32_t k_sm = smem_u32(cp_sm), q_sm = k_sm + k_room;
  float* A = reinterpret_cast<float*>(cp_sm + k_room + q_room);
  float* Ti = reinterpret_cast<float*>(cp_sm + k_room);
  {
    const __nv_bfloat16* src = p.act + static_cast<size_t>(t0) * p.ld + qh * p.dim;
    TileLoader(p.dim, p.ld, tid, kChunkThreads).load(k_sm, q_sm - k_sm, src + p.k_off, src + p.q_off, cnt, ldk);
  }
  if (tid < kBlk) {  // decays, their logarithms (base 2) summed up; a decay of 0 becomes 2^-1000
    float lg = 0.f, beta = 0.f;
    if (tid < cnt) {
      if (DELTA) {
        const float* ba = p.ba + static_cast<size_t>(t0 + tid) * 2 * p.heads;
        beta = sigmoid_of(ba[h]);
        lg = chunk_log_decay(p.a_log[h], ba[p.heads + h], p.dt_bias[h]);
      } else {
        lg = logf(p.decay[h]);
      }
      lg = fmaxf(lg * 1.4426950408889634f, -1000.f);
    }
#pragma unroll
    for (int s = 1; s < 32; s <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, lg, s);
      if (lane >= s) lg += y;
    }
    L[tid] = lg;
    bt[tid] = beta;
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  const float carry = L[31];
  if (DELTA) {
    // two threads per row
    const int r = tid >> 1;
    const uint8_t* kr = cp_sm + r * ldk * 2;
    const uint8_t* qr = cp_sm + k_room + r * ldk * 2;
    float kk = 0.f, qq = 0.f;
    for (int c = tid & 1; c < p.dim / 8; c += 2) {
      float a[8], b[8];
      load8<__nv_bfloat16>(reinterpret_cast<const __nv_bfloat16*>(kr) + c * 8, a);
      load8<__nv_bfloat16>(reinterpret_cast<const __nv_bfloat16*>(qr) + c * 8, b);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        kk = fmaf(a[e], a[e], kk);
        qq = fmaf(b[e], b[e], qq);
      }
    }
    kk += __shfl_xor_sync(0xffffffffu, kk, 1);
    qq += __shfl_xor_sync(0xffffffffu, qq, 1);
    if ((tid & 1) == 0) {
      ikv[r] = 1.f / sqrtf(kk + 1e-6f);
      iqv[r] = p.q_scale / sqrtf(qq + 1e-6f);
    }
  } else if (tid < kBlk) {
    ikv[tid] = 1.f;
    iqv[tid] = p.q_scale;
  }
  __syncthreads();
  if (tid >= 32 && tid < kBlk) L[tid] += carry;
  __syncthreads();
  const size_t bh = static_cast<size_t>(blk) * p.heads + h;
  {
    float* f = p.factors + bh * kFactors * kBlk;
    const float last = L[kBlk - 1];
    if (tid < kBlk) {
      const float G = exp2f(L[tid]);
      f[tid] = G * iqv[tid];
      f[kBlk + tid] = G * ikv[tid];
      f[2 * kBlk + tid] = bt[tid];
      f[3 * kBlk + tid] = exp2f(last - L[tid]) * ikv[tid];
    }
    if (tid == 0) p.factors[static_cast<size_t>(p.blocks) * p.heads * kFactors * kBlk + bh] = exp2f(last);
  }
  // rows 16 warp.. of Q K^T and K K^T, columns up to the diagonal
  float sq[8][4], sk[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) sq[n][e] = sk[n][e] = 0.f;
  for (int ks = 0; ks < p.dim / 16; ++ks) {
    uint32_t aq[4], ak[4];
    const uint32_t a_off = ((warp * 16 + (lj & 1) * 8 + lr) * ldk + ks * 16 + (lj >> 1) * 8) * 2;
    ldmatrix_x4(q_sm + a_off, aq[0], aq[1], aq[2], aq[3]);
    if (DELTA) ldmatrix_x4(k_sm + a_off, ak[0], ak[1], ak[2], ak[3]);
#pragma unroll
    for (int n2 = 0; n2 < 4; ++n2) {
      if (n2 > warp) break;
      uint32_t b0, b1, b2, b3;  // keys 16 n2.. + 8
      ldmatrix_x4(k_sm + ((n2 * 16 + (lj >> 1) * 8 + lr) * ldk + ks * 16 + (lj & 1) * 8) * 2, b0, b1, b2, b3);
      mma_bf16_16816(sq[2 * n2], aq, b0, b1);
      mma_bf16_16816(sq[2 * n2 + 1], aq, b2, b3);
      if (DELTA) {
        mma_bf16_16816(sk[2 * n2], ak, b0, b1);
        mma_bf16_16816(sk[2 * n2 + 1], ak, b2, b3);
      }
    }
  }
  const int r0 = warp * 16 + gq, r1 = r0 + 8;
#pragma unroll
  for (int n = 0; n < 8; ++n) {
    if (n > 2 * warp + 1) break;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = e < 2 ? r0 : r1, s = n * 8 + 2 * tq + (e & 1);
      const float w = s <= t ? fast_ex2(L[t] - L[s]) * ikv[s] : 0.f;
      sq[n][e] *= w * iqv[t];
      if (DELTA) A[t * 68 + s] = s < t ? sk[n][e] * w * ikv[t] * bt[t] : 0.f;
    }
  }
  uint4* pf = p.p_frags + bh * kFragsPerBlock + warp * (4 * 2 * 32) + lane;
#pragma unroll
  for (int ks = 0; ks < 4; ++ks) {
    if (ks > warp) break;
    uint4 hi, lo;
    split2(sq[2 * ks][0], sq[2 * ks][1], hi.x, lo.x);
    split2(sq[2 * ks][2], sq[2 * ks][3], hi.y, lo.y);
    split2(sq[2 * ks + 1][0], sq[2 * ks + 1][1], hi.z, lo.z);
    split2(sq[2 * ks + 1][2], sq[2 * ks + 1][3], hi.w, lo.w);
    pf[ks * 64] = hi;
    pf[ks * 64 + 32] = lo;
  }
  if (!DELTA) return;
  __syncthreads();
  // (I + A)^-1: a warp inverts its 16 x 16 block on the diagonal, a column per lane; then twice [[X, 0], [-Y A' X, Y]] joins
  // neighbours of 16 and of 32.  Zeros above the diagonal are written where the joins read them.
  {
    const float* Ad = A + warp * 16 * 68 + warp * 16;
    float* Td = Ti + warp * 16 * 68 + warp * 16;
    if (lane < 16) {
      float x[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float a0 = i == lane ? 1.f : 0.f, a1 = 0.f;
#pragma unroll
        for (int s = 0; s < i; s += 2) {
          const float2 a = *reinterpret_cast<const float2*>(Ad + i * 68 + s);
          a0 = fmaf(-a.x, x[s], a0);
          if (s + 1 < i) a1 = fmaf(-a.y, x[s + 1], a1);
        }
        x[i] = a0 + a1;
        Td[i * 68 + lane] = x[i];
      }
    } else if (warp < 3) {  // the 16 columns to the right
      for (int i = 0; i < 16; ++i) Td[i * 68 + lane] = 0.f;
    }
  }
  float* tmp = reinterpret_cast<float*>(cp_sm);  // [32][68]
  __syncthreads();
  {
    const int pair = warp >> 1, at = pair * 32, t = tid & 63;
    float* tp = tmp + pair * 16 * 68;
    small_product<16>(A + (at + 16) * 68 + at, Ti + at * 68 + at, tp, 1.f, t, 64);
    __syncthreads();
    small_product<16>(Ti + (at + 16) * 68 + at + 16, tp, Ti + (at + 16) * 68 + at, -1.f, t, 64);
  }
  __syncthreads();
  small_product<32>(A + 32 * 68, Ti, tmp, 1.f, tid, kChunkThreads);
  __syncthreads();
  small_product<32>(Ti + 32 * 68 + 32, tmp, Ti + 32 * 68, -1.f, tid, kChunkThreads);
  __syncthreads();
  uint4* tf = p.t_frags + bh * kFragsPerBlock + warp * (4 * 2 * 32) + lane;
#pragma unroll
  for (int ks = 0; ks < 4; ++ks) {
    if (ks > warp) break;
    const float2 a = *reinterpret_cast<const float2*>(Ti + r0 * 68 + ks * 16 + 2 * tq);
    const float2 b = *reinterpret_cast<const float2*>(Ti + r1 * 68 + ks * 16 + 2 * tq);
    const float2 c = *reinterpret_cast<const float2*>(Ti + r0 * 68 + ks * 16 + 8 + 2 * tq);
    const float2 d = *reinterpret_cast<const float2*>(Ti + r1 * 68 + ks * 16 + 8 + 2 * tq);
    uint4 hi, lo;
    split2(a.x, a.y, hi.x, lo.x);
    split2(b.x, b.y, hi.y, lo.y);
    split2(c.x, c.y, hi.z, lo.z);
    split2(d.x, d.y, hi.w, lo.w);
    tf[ks * 64] = hi;
    tf[ks * 64 + 32] = lo;
  }
}

// B operand [16 rows][16 columns] of a row-major tile: columns 0-7 in b[0], b[1], 8-15 in b[2], b[3].
__device__ __forceinline__ void load_b16(uint32_t tile, int row, int lane, uint32_t (&b)[4]) {
  const int lj = lane >> 3, lr = lane & 7;
  ldmatrix_x4_trans(tile + ((row + lr + (lj & 1) * 8) * kSmLd + (lj >> 1) * 8) * 2, b[0], b[1], b[2], b[3]);
}
__device__ __forceinline__ void mma_2(float (&d)[2][4], const uint32_t (&a)[4], const uint32_t (&b)[4]) {
  mma_bf16_16816(d[0], a, b[0], b[1]);
  mma_bf16_16816(d[1], a, b[2], b[3]);
}
__device__ __forceinline__ void get4(const uint4& v, uint32_t (&a)[4]) {
  a[0] = v.x;
  a[1] = v.y;
  a[2] = v.z;
  a[3] = v.w;
}

constexpr int kScanThreads = 9 * 32;
constexpr int kTileChunk = kBlk * 128;  // 64 tokens x 64 columns, 128-byte swizzle

// Warps 0-3 carry the state (16 tokens each of K S, the residuals and U; MT 16-row tiles each of the state), warps 4-7 make the
// output (16 tokens each) while the state moves on, warp 8 asks for the next block's k and q by TMA in boxes of 64 tokens x 64
// columns (past a head's size they bring the next one's columns, which nobody reads; past the last token zeros).  All warps meet
// at two or three barriers per block: state in place, residuals in place, U in place.
template <int MT, bool DELTA, int CTAS>
__global__ void __launch_bounds__(kScanThreads, CTAS)
chunk_scan_kernel(const __grid_constant__ CUtensorMap act_map, const ChunkParams p) {
  extern __shared__ uint8_t cs_raw[];
  __shared__ __align__(8) uint64_t bar_mem[2];
  const uint32_t cs_base = (smem_u32(cs_raw) + 1023u) & ~1023u;
  uint8_t* cs_sm = cs_raw + (cs_base - smem_u32(cs_raw));
  const uint32_t bars = smem_u32(bar_mem);
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&act_map);
    mbar_init(bars, 1);
    mbar_init(bars + 8, 1);
    fence_mbar_init();
    fence_proxy_async();
  }
  __syncthreads();
  grid_dep_wait();
  grid_dep_launch();
  const int h = blockIdx.y, c0 = blockIdx.x * 16, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, tq = lane & 3, lj = lane >> 3, lr = lane & 7;
  const int qh = h / (p.heads / p.qk_heads), chunks = (p.dim + 63) / 64, tile_bytes = chunks * kTileChunk, mtiles = p.dim / 16;
  const int first = p.positions[0], slot = p.slots[0];
  if (slot < 0 || slot >= p.num_slots || first < 0) {
    if (tid == 0) set_error(p.err, kErrDevBadBlockId);
    return;
  }
  const uint32_t kq_sm = cs_base;                       // [2 buffers][k, q][chunks][64 tokens][128 bytes]
  const uint32_t s_sm = kq_sm + 4 * tile_bytes;         // state: [high, low][dim][kSmLd]
  const uint32_t s_lo = p.dim * kSmLd * 2;
  const uint32_t u_sm = s_sm + 2 * s_lo;                // residuals, U, scaled U: [3][high, low][64][kSmLd]
  constexpr uint32_t kURows = kBlk * kSmLd * 2;
  uint8_t* s_ptr = cs_sm + 4 * tile_bytes;
  uint8_t* u_ptr = s_ptr + 2 * s_lo;
  const size_t fac_total = static_cast<size_t>(p.blocks) * p.heads * kFactors * kBlk;

  if (warp == 8) {
    // --------------------------------------------------------------- loader --
#pragma unroll 1
    for (int blk = -1; blk < p.blocks; ++blk) {
      if (blk >= 0) __syncthreads();  // everybody is through with the other tiles
      if (lane == 0 && blk + 1 < p.blocks) {
        const uint32_t bar = bars + 8 * ((blk + 1) & 1), dst = kq_sm + ((blk + 1) & 1) * 2 * tile_bytes;
        mbar_arrive_expect_tx(bar, 2 * tile_bytes);
        for (int c = 0; c < chunks; ++c) {
          tma_load_2d(dst + c * kTileChunk, &act_map, bar, p.k_off + qh * p.dim + c * 64, (blk + 1) * kBlk);
          tma_load_2d(dst + tile_bytes + c * kTileChunk, &act_map, bar, p.q_off + qh * p.dim + c * 64, (blk + 1) * kBlk);
        }
      }
      __syncwarp();
      if (blk < 0) continue;
      if (DELTA) __syncthreads();
      __syncthreads();
    }
    return;
  }
  bool alive = true;
  const int w4 = warp & 3, r0 = w4 * 16 + gq, r1 = r0 + 8;
  // A operand of 16 tokens: 16 columns further is ^ 32, ^ 64, ^ 96 inside a chunk
  const uint32_t a_off = swz128(w4 * 16 + (lj & 1) * 8 + lr, lj >> 1);

  if (warp >= 4) {
    // --------------------------------------------------------------- output --
#pragma unroll 1
    for (int blk = 0; blk < p.blocks; ++blk) {
      const int t0 = blk * kBlk, cnt = min(kBlk, p.rows - t0);
      const size_t bh = static_cast<size_t>(blk) * p.heads + h;
      const float* fac = p.factors + bh * kFactors * kBlk;
      const float gq0 = fac[r0], gq1 = fac[r1];
      const uint4* pf = p.p_frags + bh * kFragsPerBlock + w4 * (4 * 2 * 32) + lane;
      uint4 pfr[4][2];
#pragma unroll
      for (int ks = 0; ks < 4; ++ks)
        if (ks <= w4) {
          pfr[ks][0] = __ldg(pf + ks * 64);
          pfr[ks][1] = __ldg(pf + ks * 64 + 32);
        }
      float Q[2][2][4];  // from the state's high and low parts
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) Q[0][n][e] = Q[1][n][e] = 0.f;
      __syncthreads();  // state in place
      if (alive) alive = mbar_wait(bars + 8 * (blk & 1), (blk >> 1) & 1, p.err);
      const uint32_t q_sm = kq_sm + (blk & 1) * 2 * tile_bytes + tile_bytes;
#pragma unroll 4
      for (int ks = 0; ks < mtiles; ++ks) {
        uint32_t bh4[4], bl4[4], a[4];
        load_b16(s_sm, ks * 16, lane, bh4);
        load_b16(s_sm + s_lo, ks * 16, lane, bl4);
        ldmatrix_x4(q_sm + (ks >> 2) * kTileChunk + (a_off ^ ((ks & 3) * 32)), a[0], a[1], a[2], a[3]);
        mma_2(Q[0], a, bh4);
        mma_2(Q[1], a, bl4);
      }
      if (DELTA) __syncthreads();  // residuals in place
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          Q[0][n][e] = (Q[0][n][e] + Q[1][n][e]) * (e < 2 ? gq0 : gq1);
          Q[1][n][e] = 0.f;
        }
      __syncthreads();  // U in place
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks > w4) break;
        uint32_t bh4[4], bl4[4], a[4], al[4];
        load_b16(u_sm + 2 * kURows, ks * 16, lane, bh4);
        get4(pfr[ks][0], a);
        get4(pfr[ks][1], al);
        mma_2(Q[0], a, bh4);
        mma_2(Q[1], al, bh4);
        if (DELTA) {  // v is exactly bf16
          load_b16(u_sm + 3 * kURows, ks * 16, lane, bl4);
          mma_2(Q[0], a, bl4);
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int r = e == 0 ? r0 : r1;
          if (r < cnt)
            *reinterpret_cast<float2*>(p.o + (static_cast<size_t>(t0 + r) * p.heads + h) * p.vdim + c0 + n * 8 + 2 * tq) =
                make_float2(Q[0][n][e] + Q[1][n][e], Q[0][n][e + 1] + Q[1][n][e + 1]);
        }
    }
    return;
  }

  // ------------------------------------------------------------------ state --
  const size_t half = static_cast<size_t>(p.heads) * p.dim * p.vdim;
  float* st = p.state + static_cast<size_t>(slot) * 2 * half + static_cast<size_t>(h) * p.dim * p.vdim + c0;
  float S[MT][2][4];
  {
    const float* src = st + ((first - 1) & 1) * half;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int mt = warp + 4 * i, r = mt * 16 + gq + (e >> 1) * 8;
          float2 v = make_float2(0.f, 0.f);
          if (first > 0 && mt < mtiles) v = *reinterpret_cast<const float2*>(src + static_cast<size_t>(r) * p.vdim + n * 8 + 2 * tq);
          S[i][n][e] = v.x;
          S[i][n][e + 1] = v.y;
        }
  }
#pragma unroll 1
  for (int blk = 0; blk < p.blocks; ++blk) {
    // the state as an operand
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int mt = warp + 4 * i;
      if (mt >= mtiles) break;
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          uint32_t hi, lo;
          split2(S[i][n][e], S[i][n][e + 1], hi, lo);
          const uint32_t at = ((mt * 16 + gq + (e >> 1) * 8) * kSmLd + n * 8 + 2 * tq) * 2;
          *reinterpret_cast<uint32_t*>(s_ptr + at) = hi;
          *reinterpret_cast<uint32_t*>(s_ptr + s_lo + at) = lo;
        }
    }
    const int t0 = blk * kBlk, cnt = min(kBlk, p.rows - t0);
    const size_t bh = static_cast<size_t>(blk) * p.heads + h;
    // inputs that go to registers
    const float* fac = p.factors + bh * kFactors * kBlk;
    const float uk0 = fac[3 * kBlk + r0], uk1 = fac[3 * kBlk + r1];
    const float g_all = p.factors[fac_total + bh];
    float v[2][4], gk0 = 0.f, gk1 = 0.f, be0 = 0.f, be1 = 0.f;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int r = e == 0 ? r0 : r1;
        float2 f = make_float2(0.f, 0.f);
        if (r < cnt)
          f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p.act + static_cast<size_t>(t0 + r) * p.ld + p.v_off + h * p.vdim + c0 + n * 8 + 2 * tq));
        v[n][e] = f.x;
        v[n][e + 1] = f.y;
      }
    uint4 tfr[4][2];
    if (DELTA) {
      gk0 = fac[kBlk + r0];
      gk1 = fac[kBlk + r1];
      be0 = fac[2 * kBlk + r0];
      be1 = fac[2 * kBlk + r1];
      const uint4* tf = p.t_frags + bh * kFragsPerBlock + warp * (4 * 2 * 32) + lane;
#pragma unroll
      for (int ks = 0; ks < 4; ++ks)
        if (ks <= warp) {
          tfr[ks][0] = __ldg(tf + ks * 64);
          tfr[ks][1] = __ldg(tf + ks * 64 + 32);
        }
    }
    __syncthreads();  // state in place
    if (alive) alive = mbar_wait(bars + 8 * (blk & 1), (blk >> 1) & 1, p.err);
    const uint32_t k_sm = kq_sm + (blk & 1) * 2 * tile_bytes;
    float U[2][4];
    if (DELTA) {
      float K[2][2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) K[0][n][e] = K[1][n][e] = 0.f;
#pragma unroll 4
      for (int ks = 0; ks < mtiles; ++ks) {
        uint32_t bh4[4], bl4[4], a[4];
        load_b16(s_sm, ks * 16, lane, bh4);
        load_b16(s_sm + s_lo, ks * 16, lane, bl4);
        ldmatrix_x4(k_sm + (ks >> 2) * kTileChunk + (a_off ^ ((ks & 3) * 32)), a[0], a[1], a[2], a[3]);
        mma_2(K[0], a, bh4);
        mma_2(K[1], a, bl4);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const float be = e == 0 ? be0 : be1, gk = e == 0 ? gk0 : gk1;
          uint32_t hi, lo;
          split2(be * (v[n][e] - gk * (K[0][n][e] + K[1][n][e])), be * (v[n][e + 1] - gk * (K[0][n][e + 1] + K[1][n][e + 1])), hi, lo);
          const uint32_t at = ((e == 0 ? r0 : r1) * kSmLd + n * 8 + 2 * tq) * 2;
          *reinterpret_cast<uint32_t*>(u_ptr + at) = hi;
          *reinterpret_cast<uint32_t*>(u_ptr + kURows + at) = lo;
          K[0][n][e] = K[0][n][e + 1] = K[1][n][e] = K[1][n][e + 1] = 0.f;
        }
      __syncthreads();  // residuals in place
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks > warp) break;
        uint32_t bh4[4], bl4[4], a[4], al[4];
        load_b16(u_sm, ks * 16, lane, bh4);
        load_b16(u_sm + kURows, ks * 16, lane, bl4);
        get4(tfr[ks][0], a);
        get4(tfr[ks][1], al);
        mma_2(K[0], a, bh4);
        mma_2(K[1], a, bl4);
        mma_2(K[1], al, bh4);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) U[n][e] = K[0][n][e] + K[1][n][e];
    } else {
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) U[n][e] = v[n][e];
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const float uk = e == 0 ? uk0 : uk1;
        uint32_t hi, lo;
        const uint32_t at = ((e == 0 ? r0 : r1) * kSmLd + n * 8 + 2 * tq) * 2;
        split2(U[n][e], U[n][e + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(u_ptr + 2 * kURows + at) = hi;
        if (DELTA) *reinterpret_cast<uint32_t*>(u_ptr + 3 * kURows + at) = lo;
        split2(U[n][e] * uk, U[n][e + 1] * uk, hi, lo);
        *reinterpret_cast<uint32_t*>(u_ptr + 4 * kURows + at) = hi;
        *reinterpret_cast<uint32_t*>(u_ptr + 5 * kURows + at) = lo;
      }
    __syncthreads();  // U in place
    // the state moves on
    float D[MT][2][4];  // from U's low part
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          S[i][n][e] *= g_all;
          D[i][n][e] = 0.f;
        }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t bh4[4], bl4[4];
      load_b16(u_sm + 4 * kURows, ks * 16, lane, bh4);
      load_b16(u_sm + 5 * kURows, ks * 16, lane, bl4);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const int mt = warp + 4 * i;
        if (mt >= mtiles) break;
        uint32_t a[4];  // K^T: rows = state rows, columns = tokens
        ldmatrix_x4_trans(k_sm + (mt >> 2) * kTileChunk + swz128(ks * 16 + lr + (lj >> 1) * 8, (mt & 3) * 2 + (lj & 1)), a[0], a[1], a[2],
                          a[3]);
        mma_2(S[i], a, bh4);
        mma_2(D[i], a, bl4);
      }
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][n][e] += D[i][n][e];
  }
  float* dst = st + ((first + p.rows - 1) & 1) * half;
#pragma unroll
  for (int i = 0; i < MT; ++i) {
    const int mt = warp + 4 * i;
    if (mt >= mtiles) break;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; e += 2)
        *reinterpret_cast<float2*>(dst + static_cast<size_t>(mt * 16 + gq + (e >> 1) * 8) * p.vdim + n * 8 + 2 * tq) =
            make_float2(S[i][n][e], S[i][n][e + 1]);
  }
}

struct ChunkWorkspace {
  size_t t_frags, factors, total;
};
static ChunkWorkspace chunk_carve(int rows, int heads, bool delta) {
  const size_t bh = static_cast<size_t>((rows + kBlk - 1) / kBlk) * heads;
  ChunkWorkspace w;
  w.t_frags = bh * kFragsPerBlock * 16;
  w.factors = w.t_frags * (delta ? 2 : 1);
  w.total = w.factors + bh * (kFactors * kBlk + 1) * 4;
  return w;
}

template <bool DELTA>
static int launch_chunks(const ChunkParams& p, cudaStream_t st) {
  const size_t prep = prep_k_bytes(p.dim) + prep_q_bytes(p.dim, DELTA) + (DELTA ? kBlk * 68 * 4 : 0);
  const size_t scan = 1024 + 4 * static_cast<size_t>((p.dim + 63) / 64) * kTileChunk + (2 * p.dim + 6 * kBlk) * kSmLd * 2;
  CUtensorMap act_map;
  int rc = get_tensor_map_2d(p.act, p.rows, p.ld, 2, kBlk, 64, &act_map);
  if (rc) return rc;
  rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&chunk_prepare_kernel<DELTA>), 128 * 1024);
  if (rc) return rc;
  B200_CUDA(launch_overlapped(chunk_prepare_kernel<DELTA>, dim3(p.blocks, p.heads), dim3(kChunkThreads), prep, st, p));
  const dim3 grid(p.vdim / 16, p.heads);
  int sms = 0;
  rc = device_sm_count(&sms);
  if (rc) return rc;
  const bool two = static_cast<int>(grid.x * grid.y) > sms;  // two CTAs per SM cost registers
#define B200_CHUNK(MT, CTAS)                                                                                       \
  do {                                                                                                             \
    rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&chunk_scan_kernel<MT, DELTA, CTAS>), 110 * 1024);       \
    if (rc) return rc;                                                                                             \
    B200_CUDA(launch_overlapped(chunk_scan_kernel<MT, DELTA, CTAS>, grid, dim3(kScanThreads), scan, st, act_map, p)); \
  } while (0)
  if (p.dim <= 64 && two) B200_CHUNK(1, 2);
  else if (p.dim <= 64) B200_CHUNK(1, 1);
  else if (two) B200_CHUNK(2, 2);
  else B200_CHUNK(2, 1);
#undef B200_CHUNK
  return 0;
}

}  // namespace b200

using namespace b200;

extern "C" size_t b200_state_chunk_workspace_bytes(int num_rows, int heads, int delta) {
  return num_rows > 0 && heads > 0 ? chunk_carve(num_rows, heads, delta != 0).total : 16;
}

extern "C" int b200_state_chunk(const void* act, int ld, int q_off, int k_off, int v_off, const float* ba, const float* a_log,
                                const float* dt_bias, const float* decay, float* state, const int32_t* slots,
                                const int32_t* positions, float* o, void* workspace, size_t workspace_bytes, void* status_word,
                                int num_rows, int heads, int qk_heads, int dim, int vdim, int num_slots, float q_scale,
                                void* stream) {
  B200_REQUIRE(act && state && slots && positions && o && workspace, "state_chunk: null pointer");
  B200_REQUIRE((decay != nullptr) != (ba && a_log && dt_bias), "state_chunk: a fixed decay, or beta, a_log and dt_bias");
  B200_REQUIRE(num_rows > 0 && heads > 0 && heads <= 65535 && qk_heads > 0 && heads % qk_heads == 0 && dim > 0 && dim <= 128 &&
                   dim % 16 == 0 && vdim > 0 && vdim % 16 == 0 && num_slots > 0,
               "state_chunk: %d rows, %d heads over %d, state %d x %d (multiples of 16, at most 128 rows)", num_rows, heads, qk_heads,
               dim, vdim);
  B200_REQUIRE(q_off >= 0 && k_off >= 0 && v_off >= 0 && q_off + qk_heads * dim <= ld && k_off + qk_heads * dim <= ld &&
                   v_off + heads * vdim <= ld && (ld | q_off | k_off | v_off) % 8 == 0,
               "state_chunk: q, k and v do not fit rows of %d", ld);
  B200_REQUIRE(aligned16({act, state, o, workspace}), "state_chunk: buffers must be 16-byte aligned");
  const ChunkWorkspace w = chunk_carve(num_rows, heads, decay == nullptr);
  if (workspace_bytes < w.total) {
    set_detail("state_chunk: workspace %zu < required %zu", workspace_bytes, w.total);
    return -kErrWorkspace;
  }
  int rc = check_device(nullptr);
  if (rc) return rc;
  uint8_t* ws = static_cast<uint8_t*>(workspace);
  const ChunkParams p{static_cast<const __nv_bfloat16*>(act), ld, q_off, k_off, v_off, ba, a_log, dt_bias, decay, state, slots,
                      positions, o, reinterpret_cast<uint4*>(ws), reinterpret_cast<uint4*>(ws + (decay ? 0 : w.t_frags)),
                      reinterpret_cast<float*>(ws + w.factors), static_cast<int*>(status_word), num_rows,
                      (num_rows + kBlk - 1) / kBlk, heads, qk_heads, dim, vdim, num_slots, q_scale};
  return decay ? launch_chunks<false>(p, as_stream(stream)) : launch_chunks<true>(p, as_stream(stream));
}
