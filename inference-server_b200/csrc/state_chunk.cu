// The recurrences of state_scan.cu for a chunk of prompt tokens of one sequence, 64 tokens at a time on the tensor cores
// (mma.sync), bf16 activations, dim and vdim multiples of 16, dim at most 128.
//
// With G_t the product of the block's decays up to token t and S the state before the block (rows of q, k are raw; iq_t, ik_t
// are the factors that make them unit vectors, q's scale included, or 1):
//     P[t, s] = iq_t ik_s G_t / G_s (q_t . k_s),  s <= t            A[t, s] = beta_t ik_t ik_s G_t / G_s (k_t . k_s),  s < t
//     U = (I + A)^-1 diag(beta) (V - diag(G ik) K S)    (gated delta rule; otherwise U = V)
//     O = diag(G iq) Q S + P U                           S' = G_64 S + K^T diag(G_64 / G ik) U
// The prepare kernel makes P and T = (I + A)^-1 for all blocks and heads side by side (the inverse by forward substitution, a
// column per thread); the block kernel walks the blocks in order, a CTA per head and 16 columns of the state, which stay in
// registers as accumulators.
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

// A 64-row tile of q or k into shared memory, rows of dim + 8, zero rows past the last token.
__device__ __forceinline__ void load_tile(uint32_t dst, const __nv_bfloat16* src, int ld, int cnt, int dim) {
  const int pieces = dim / 8;
  for (int i = threadIdx.x; i < kBlk * pieces; i += kChunkThreads) {
    const int r = i / pieces, c = i - r * pieces;
    cp_async16(dst + (r * (dim + 8) + c * 8) * 2, src + static_cast<size_t>(r < cnt ? r : 0) * ld + c * 8, r < cnt);
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
  const uint32_t k_sm = smem_u32(cp_sm), q_sm = k_sm + kBlk * ldk * 2;
  float* A = reinterpret_cast<float*>(cp_sm + 2 * kBlk * ldk * 2);  // [64][68]
  float* Ti = A + kBlk * 68;
  load_tile(k_sm, p.act + static_cast<size_t>(t0) * p.ld + p.k_off + qh * p.dim, p.ld, cnt, p.dim);
  load_tile(q_sm, p.act + static_cast<size_t>(t0) * p.ld + p.q_off + qh * p.dim, p.ld, cnt, p.dim);
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (tid < kBlk) {  // decays, summed up in the log domain; a decay of 0 becomes e^-1000
    float lg = 0.f, beta = 0.f;
    if (tid < cnt) {
      if (DELTA) {
        const float* ba = p.ba + static_cast<size_t>(t0 + tid) * 2 * p.heads;
        beta = sigmoid_of(ba[h]);
        lg = chunk_log_decay(p.a_log[h], ba[p.heads + h], p.dt_bias[h]);
      } else {
        lg = logf(p.decay[h]);
      }
      lg = fmaxf(lg, -1000.f);
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
    const __nv_bfloat16* kp = reinterpret_cast<const __nv_bfloat16*>(cp_sm);
    for (int r = warp * 16; r < warp * 16 + 16; ++r) {
      float kk = 0.f, qq = 0.f;
      for (int c = lane; c < p.dim; c += 32) {
        const float a = __bfloat162float(kp[r * ldk + c]), b = __bfloat162float(kp[(kBlk + r) * ldk + c]);
        kk = fmaf(a, a, kk);
        qq = fmaf(b, b, qq);
      }
      kk = warp_sum(kk);
      qq = warp_sum(qq);
      if (lane == 0) {
        ikv[r] = 1.f / sqrtf(kk + 1e-6f);
        iqv[r] = p.q_scale / sqrtf(qq + 1e-6f);
      }
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
      const float G = expf(L[tid]);
      f[tid] = G * iqv[tid];
      f[kBlk + tid] = G * ikv[tid];
      f[2 * kBlk + tid] = bt[tid];
      f[3 * kBlk + tid] = expf(last - L[tid]) * ikv[tid];
    }
    if (tid == 0) p.factors[static_cast<size_t>(p.blocks) * p.heads * kFactors * kBlk + bh] = expf(last);
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
      const float w = s <= t ? expf(L[t] - L[s]) * ikv[s] : 0.f;
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
  if (tid < kBlk) {  // column tid of the inverse
    float x[kBlk];
#pragma unroll
    for (int i = 0; i < kBlk; ++i) {
      float a0 = i == tid ? 1.f : 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
      for (int s = 0; s < i; s += 4) {
        const float4 a = *reinterpret_cast<const float4*>(A + i * 68 + s);
        a0 = fmaf(-a.x, x[s], a0);
        if (s + 1 < i) a1 = fmaf(-a.y, x[s + 1], a1);
        if (s + 2 < i) a2 = fmaf(-a.z, x[s + 2], a2);
        if (s + 3 < i) a3 = fmaf(-a.w, x[s + 3], a3);
      }
      x[i] = (a0 + a1) + (a2 + a3);
      Ti[i * 68 + tid] = x[i];
    }
  }
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

// MT: 16-row tiles of the state per warp.
template <int MT, bool DELTA>
__global__ void __launch_bounds__(kChunkThreads)
chunk_scan_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) uint8_t cs_sm[];
  grid_dep_wait();
  grid_dep_launch();
  const int h = blockIdx.y, c0 = blockIdx.x * 16, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int gq = lane >> 2, tq = lane & 3, lj = lane >> 3, lr = lane & 7;
  const int qh = h / (p.heads / p.qk_heads), ldk = p.dim + 8, tile_bytes = kBlk * ldk * 2, mtiles = p.dim / 16;
  const int first = p.positions[0], slot = p.slots[0];
  if (slot < 0 || slot >= p.num_slots || first < 0) {
    if (tid == 0) set_error(p.err, kErrDevBadBlockId);
    return;
  }
  const uint32_t kq_sm = smem_u32(cs_sm);               // [2 buffers][k, q][64][ldk]
  const uint32_t s_sm = kq_sm + 4 * tile_bytes;         // state: [high, low][dim][kSmLd]
  const uint32_t s_lo = p.dim * kSmLd * 2;
  const uint32_t u_sm = s_sm + 2 * s_lo;                // residuals / U / scaled U: [3][high, low][64][kSmLd]
  constexpr uint32_t kURows = kBlk * kSmLd * 2;
  uint8_t* u_ptr = cs_sm + 4 * tile_bytes + 2 * s_lo;
  uint8_t* s_ptr = cs_sm + 4 * tile_bytes;
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
  auto fetch = [&](int blk) {
    const int t0 = blk * kBlk, cnt = min(kBlk, p.rows - t0);
    const uint32_t dst = kq_sm + (blk & 1) * 2 * tile_bytes;
    const __nv_bfloat16* src = p.act + static_cast<size_t>(t0) * p.ld + qh * p.dim;
    load_tile(dst, src + p.k_off, p.ld, cnt, p.dim);
    load_tile(dst + tile_bytes, src + p.q_off, p.ld, cnt, p.dim);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);
  const int r0 = warp * 16 + gq, r1 = r0 + 8;
#pragma unroll 1
  for (int blk = 0; blk < p.blocks; ++blk) {
    const int t0 = blk * kBlk, cnt = min(kBlk, p.rows - t0);
    const size_t bh = static_cast<size_t>(blk) * p.heads + h;
    // this block's inputs that go to registers
    const float* fac = p.factors + bh * kFactors * kBlk;
    const float gq0 = fac[r0], gq1 = fac[r1], gk0 = fac[kBlk + r0], gk1 = fac[kBlk + r1];
    const float be0 = fac[2 * kBlk + r0], be1 = fac[2 * kBlk + r1], uk0 = fac[3 * kBlk + r0], uk1 = fac[3 * kBlk + r1];
    const float g_all = p.factors[static_cast<size_t>(p.blocks) * p.heads * kFactors * kBlk + bh];
    float v[2][4];
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
    const uint4* pf = p.p_frags + bh * kFragsPerBlock + warp * (4 * 2 * 32) + lane;
    const uint4* tf = p.t_frags + bh * kFragsPerBlock + warp * (4 * 2 * 32) + lane;
    uint4 tfr[4][2];
    if (DELTA) {
#pragma unroll
      for (int ks = 0; ks < 4; ++ks)
        if (ks <= warp) {
          tfr[ks][0] = __ldg(tf + ks * 64);
          tfr[ks][1] = __ldg(tf + ks * 64 + 32);
        }
    }
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
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // state and this block's tiles in place; everybody is through with the other tiles
    if (blk + 1 < p.blocks) fetch(blk + 1);
    const uint32_t k_sm = kq_sm + (blk & 1) * 2 * tile_bytes, q_sm = k_sm + tile_bytes;
    float KS[2][4], QS[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) KS[n][e] = QS[n][e] = 0.f;
    const uint32_t a_off = ((warp * 16 + (lj & 1) * 8 + lr) * ldk + (lj >> 1) * 8) * 2;
#pragma unroll 4
    for (int ks = 0; ks < mtiles; ++ks) {
      uint32_t bh4[4], bl4[4], a[4];
      load_b16(s_sm, ks * 16, lane, bh4);
      load_b16(s_sm + s_lo, ks * 16, lane, bl4);
      if (DELTA) {
        ldmatrix_x4(k_sm + a_off + ks * 32, a[0], a[1], a[2], a[3]);
        mma_2(KS, a, bh4);
        mma_2(KS, a, bl4);
      }
      ldmatrix_x4(q_sm + a_off + ks * 32, a[0], a[1], a[2], a[3]);
      mma_2(QS, a, bh4);
      mma_2(QS, a, bl4);
    }
    uint4 pfr[4][2];
#pragma unroll
    for (int ks = 0; ks < 4; ++ks)
      if (ks <= warp) {
        pfr[ks][0] = __ldg(pf + ks * 64);
        pfr[ks][1] = __ldg(pf + ks * 64 + 32);
      }
    float U[2][4];
    if (DELTA) {
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const float be = e == 0 ? be0 : be1, gk = e == 0 ? gk0 : gk1;
          uint32_t hi, lo;
          split2(be * (v[n][e] - gk * KS[n][e]), be * (v[n][e + 1] - gk * KS[n][e + 1]), hi, lo);
          const uint32_t at = ((e == 0 ? r0 : r1) * kSmLd + n * 8 + 2 * tq) * 2;
          *reinterpret_cast<uint32_t*>(u_ptr + at) = hi;
          *reinterpret_cast<uint32_t*>(u_ptr + kURows + at) = lo;
          U[n][e] = U[n][e + 1] = 0.f;
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
        mma_2(U, a, bh4);
        mma_2(U, a, bl4);
        mma_2(U, al, bh4);
      }
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
        *reinterpret_cast<uint32_t*>(u_ptr + 3 * kURows + at) = lo;
        split2(U[n][e] * uk, U[n][e + 1] * uk, hi, lo);
        *reinterpret_cast<uint32_t*>(u_ptr + 4 * kURows + at) = hi;
        *reinterpret_cast<uint32_t*>(u_ptr + 5 * kURows + at) = lo;
      }
    __syncthreads();  // U in place
    // state: rows of this warp's tiles
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][n][e] *= g_all;
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
        ldmatrix_x4_trans(k_sm + ((ks * 16 + lr + (lj >> 1) * 8) * ldk + mt * 16 + (lj & 1) * 8) * 2, a[0], a[1], a[2], a[3]);
        mma_2(S[i], a, bh4);
        mma_2(S[i], a, bl4);
      }
    }
    // output
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      QS[n][0] *= gq0;
      QS[n][1] *= gq0;
      QS[n][2] *= gq1;
      QS[n][3] *= gq1;
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      if (ks > warp) break;
      uint32_t bh4[4], bl4[4], a[4], al[4];
      load_b16(u_sm + 2 * kURows, ks * 16, lane, bh4);
      get4(pfr[ks][0], a);
      get4(pfr[ks][1], al);
      mma_2(QS, a, bh4);
      mma_2(QS, al, bh4);
      if (DELTA) {  // v is exactly bf16
        load_b16(u_sm + 3 * kURows, ks * 16, lane, bl4);
        mma_2(QS, a, bl4);
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int r = e == 0 ? r0 : r1;
        if (r < cnt)
          *reinterpret_cast<float2*>(p.o + (static_cast<size_t>(t0 + r) * p.heads + h) * p.vdim + c0 + n * 8 + 2 * tq) =
              make_float2(QS[n][e], QS[n][e + 1]);
      }
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
  const size_t tile = static_cast<size_t>(kBlk) * (p.dim + 8) * 2;
  const size_t prep = 2 * tile + (DELTA ? 2 * kBlk * 68 * 4 : 0), scan = 4 * tile + 2 * static_cast<size_t>(p.dim) * kSmLd * 2 + 6 * kBlk * kSmLd * 2;
  int rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&chunk_prepare_kernel<DELTA>), 128 * 1024);
  if (rc) return rc;
  B200_CUDA(launch_overlapped(chunk_prepare_kernel<DELTA>, dim3(p.blocks, p.heads), dim3(kChunkThreads), prep, st, p));
  const dim3 grid(p.vdim / 16, p.heads);
#define B200_CHUNK(MT)                                                                                           \
  do {                                                                                                           \
    rc = ensure_dynamic_smem(reinterpret_cast<const void*>(&chunk_scan_kernel<MT, DELTA>), 128 * 1024);          \
    if (rc) return rc;                                                                                           \
    B200_CUDA(launch_overlapped(chunk_scan_kernel<MT, DELTA>, grid, dim3(kChunkThreads), scan, st, p));          \
  } while (0)
  if (p.dim <= 64) B200_CHUNK(1);
  else B200_CHUNK(2);
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
