// Device-side helpers shared by the decode hot-path kernels (sm_100a only).
//
// Everything here is a thin wrapper over one PTX instruction: mbarrier
// bookkeeping, TMA tile loads, ldmatrix / mma.sync fragments, tcgen05 MMA and
// TMEM access.  Every wait is bounded: a wait that runs out records a code in a
// caller-provided error word and returns false, so a broken pipeline ends the
// kernel instead of hanging the GPU.
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_fp8.h>
#include <cuda_runtime.h>
#include <stdint.h>

#if !defined(__CUDA_ARCH__) || (__CUDA_ARCH__ >= 1000)
#define B200_DEVICE_OK 1
#endif

namespace b200 {

// Error codes written to the device-side error word (positive) and returned by
// the C-ABI (negative).  Keep in sync with b200_strerror().
enum : int {
  kErrOk = 0,
  kErrBadArg = 1,
  kErrUnsupported = 2,
  kErrWorkspace = 3,
  kErrCuda = 4,
  kErrTensorMap = 5,
  kErrDevBadBlockId = 16,   // block_table entry outside [0, num_blocks)
  kErrDevBadCtxLen = 17,    // ctx_len outside [0, max_pages * page]
  kErrDevWaitTimeout = 18,  // a bounded mbarrier wait ran out
  kErrDevBadExpert = 19,    // expert id outside [0, E)
  kErrDevPeerTimeout = 20,  // a bounded wait for another rank's flag ran out
};

// Peer receive buffers of the expert-parallel dispatch, one entry per rank (this rank included); all null
// when rows are exchanged by a library all-to-all instead.  Row (src_rank * capacity + pos) of rank d's
// buffers holds the pos-th row that src_rank sends to d.
constexpr int kMaxEpWorld = 8;
struct EpPeers {
  uint8_t* xq[kMaxEpWorld];
  float* xs[kMaxEpWorld];
  int* id[kMaxEpWorld];
  int my_rank;
};

// Row tile consumed by the grouped GEMM: up to 128 consecutive sorted rows of
// one expert (the last tile of an expert may be short).
struct __align__(16) MoeTile {
  int expert, row0, rows, pad;
};

__device__ __forceinline__ uint32_t smem_u32(const void* p) {
  return static_cast<uint32_t>(__cvta_generic_to_shared(p));
}

// Programmatic dependent launch.  grid_dep_wait(): hold until every kernel this one depends on has completed and
// its writes are visible (returns at once when the kernel was launched the ordinary way).  Every thread calls it
// before its first access to global memory and before any return, so that "this grid has completed" always
// implies "everything before it in the stream has completed".  grid_dep_launch(): the kernel after this one may
// have its blocks placed (they hold at their own grid_dep_wait()) once every block of this grid has said so.
__device__ __forceinline__ void grid_dep_wait() {
#ifdef B200_DEVICE_OK
  asm volatile("griddepcontrol.wait;" ::: "memory");
#endif
}
__device__ __forceinline__ void grid_dep_launch() {
#ifdef B200_DEVICE_OK
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
#endif
}

__device__ __forceinline__ void set_error(int* err, int code) {
  if (err != nullptr) atomicCAS(err, 0, code);
}

// ---------------------------------------------------------------- mbarrier --
__device__ __forceinline__ void mbar_init(uint32_t bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count) : "memory");
}
__device__ __forceinline__ void fence_mbar_init() {
  asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
}
__device__ __forceinline__ void fence_proxy_async() {
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}
__device__ __forceinline__ void mbar_arrive(uint32_t bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void mbar_arrive_expect_tx(uint32_t bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes)
               : "memory");
}
__device__ __forceinline__ bool mbar_try_wait(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(ok)
      : "r"(bar), "r"(parity)
      : "memory");
  return ok != 0;
}
// Bounded wait: gives up after roughly a second and flags the error word.
__device__ __forceinline__ bool mbar_wait(uint32_t bar, uint32_t parity, int* err) {
  for (uint32_t i = 0; i < (1u << 21); ++i) {
    if (mbar_try_wait(bar, parity)) return true;
    if (i > 2048) __nanosleep(128);
  }
  set_error(err, kErrDevWaitTimeout);
  return false;
}

// --------------------------------------------------------------------- TMA --
// 2-D tiled load, global -> shared, completion counted in bytes on `bar`.
// `x` is the innermost coordinate in elements; x * element size must be a
// multiple of 16 bytes.
__device__ __forceinline__ void tma_load_2d(uint32_t dst, const CUtensorMap* map, uint32_t bar,
                                            int x, int y) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes "
      "[%0], [%1, {%3, %4}], [%2];"
      ::"r"(dst), "l"(map), "r"(bar), "r"(x), "r"(y)
      : "memory");
}
// The same for a 3-D tensor: x innermost.
__device__ __forceinline__ void tma_load_3d(uint32_t dst, const CUtensorMap* map, uint32_t bar, int x, int y, int z) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes "
      "[%0], [%1, {%3, %4, %5}], [%2];"
      ::"r"(dst), "l"(map), "r"(bar), "r"(x), "r"(y), "r"(z)
      : "memory");
}
// Plain copy global -> shared; both addresses and the size multiples of 16 bytes.
__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src),
               "r"(bytes), "r"(bar)
               : "memory");
}
__device__ __forceinline__ void tma_prefetch_desc(const CUtensorMap* map) {
  asm volatile("prefetch.tensormap [%0];" ::"l"(map) : "memory");
}

// Byte offset of (row, 16-byte chunk) inside a 128-byte-swizzled tile whose
// rows are 128 bytes long and whose base is 1024-byte aligned.
__device__ __forceinline__ uint32_t swz128(uint32_t row, uint32_t chunk16) {
  return row * 128u + (((chunk16 ^ row) & 7u) << 4);
}

// ---------------------------------------------------------- warp-level MMA --
__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t& r0, uint32_t& r1,
                                            uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1,
                                                  uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}
// D(16x8, f32) += A(16x16, bf16, row) * B(16x8, bf16, col)
__device__ __forceinline__ void mma_bf16_16816(float (&d)[4], const uint32_t (&a)[4],
                                               uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 "
      "{%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16x2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

// ---------------------------------------------------------- tcgen05 / TMEM --
__device__ __forceinline__ void tmem_alloc(uint32_t smem_dst, uint32_t ncols) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_dst),
               "r"(ncols)
               : "memory");
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc(uint32_t taddr, uint32_t ncols) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols)
               : "memory");
}
__device__ __forceinline__ void tc_fence_before() {
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
}
__device__ __forceinline__ void tc_fence_after() {
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
}
// Arrives once on `bar` when every tcgen05.mma issued so far by this thread has
// finished (implies tcgen05.fence::before_thread_sync).
__device__ __forceinline__ void tc_commit(uint32_t bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(
                   bar)
               : "memory");
}
// D[tmem] (+)= A[smem] * B[smem], e4m3 x e4m3 -> f32, one K=32 slice.
__device__ __forceinline__ void tc_mma_f8(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc,
                                          uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f8f6f4 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// 32 lanes x 32 consecutive 32-bit columns; thread i of the warp gets lane
// (warp_id % 4) * 32 + i.
__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
      "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]),
        "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]),
        "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]),
        "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]),
        "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void tmem_ld_wait() {
  asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}

// Shared-memory matrix descriptor for a K-major operand tile whose rows are
// exactly 128 bytes (one swizzle-128B span): 8-row groups are 1024 bytes apart.
__device__ __forceinline__ uint64_t umma_desc_k128(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFFu) >> 4);  // start address
  d |= static_cast<uint64_t>(1) << 16;                       // leading byte offset (unused)
  d |= static_cast<uint64_t>(1024 >> 4) << 32;               // stride byte offset
  d |= static_cast<uint64_t>(1) << 46;                       // descriptor version (sm_100)
  d |= static_cast<uint64_t>(2) << 61;                       // 128-byte swizzle
  return d;
}
// Instruction descriptor: e4m3 x e4m3 -> f32, both operands K-major.
__host__ __device__ constexpr uint32_t umma_idesc_f8(uint32_t m, uint32_t n) {
  return (1u << 4)            // accumulator f32
         | (0u << 7)          // A e4m3
         | (0u << 10)         // B e4m3
         | ((n >> 3) << 17)   // N
         | ((m >> 4) << 24);  // M
}

// ------------------------------------------------------------------- misc ---
__device__ __forceinline__ float fast_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Rows of a distance table (mixed_attn.cu): entry kDistPad + d belongs to distance d, the entries before and after the window's
// distances are +inf.
constexpr int kDistPad = 256, kDistTail = 264;
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// First token a row at position L - 1 sees when positions are cut into chunks of `chunk` (0: all of them).
__device__ __forceinline__ int first_visible(int L, int chunk) {
  return chunk > 0 && L > 0 ? (L - 1) / chunk * chunk : 0;
}
// Output gate of a (row, head): sigmoid of its fp32 logit, 1 without a gate.
__device__ __forceinline__ float head_gate(const float* gate, size_t i) {
  return gate == nullptr ? 1.f : 1.f / (1.f + expf(-gate[i]));
}
// Clamped gated unit: g * sigmoid(alpha g) * (u + shift) with g capped at `limit` and u held to +-limit; an infinite limit,
// alpha 1 and shift 0 make it silu(g) * u.
__device__ __forceinline__ float clamped_glu(float g, float u, float limit, float alpha, float shift) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + shift);
}
__device__ __forceinline__ float clamped_glu_fast(float g, float u, float limit, float alpha, float shift) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return __fdividef(g, 1.f + __expf(-alpha * g)) * (u + shift);
}
__device__ __forceinline__ float silu_of(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float sigmoid_of(float z) { return 1.f / (1.f + expf(-z)); }
// SiLU of a value that is stored as T: the fast forms are good to far more than bf16 keeps.
template <typename T>
__device__ __forceinline__ float silu_as(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-z));
  else return silu_of(z);
}
template <typename T>
__device__ __forceinline__ float to_f32(T v);
template <>
__device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
__device__ __forceinline__ uint8_t to_e4m3(float v) {
  return static_cast<uint8_t>(__nv_cvt_float_to_fp8(v, __NV_SATFINITE, __NV_E4M3));
}

}  // namespace b200
