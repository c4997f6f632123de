// The decay scan of chunk_scan.cu with chunks of 128 tokens on the 5th-generation tensor cores, for stored heads of 64 or 128
// key channels.  A CTA owns 64 value columns of one head of one sequence and walks its chunks:
//
//   G  = Q K^T                              128 tokens x 128 tokens
//   Y1 = Q S          (S in two bf16 parts)  what the state gives, times e^(c_i) per row
//   D  = K^T (w V)    (w V in two parts)     what the chunk adds to the state, w_j = e^(c_last - c_j) b_j
//   Y2 = M V          (M in two parts)       M = G e^(c_i - c_j) b_j below the diagonal
//
// with the accumulators in tensor memory.  One warp issues the products and the loads (TMA: the next chunk's k and v at the
// start of a chunk, q once Y1 is complete) and sums the next chunk's log decays behind the last product.  Three warps write
// w V (shared memory to shared memory).  Eight warps do the rest, a pair of warps per 32 rows: M (tensor memory to tensor
// memory, where it is the left operand of its product; the pair takes turns at blocks of 32 tokens), the outputs, and the
// state, which stays in their registers in fp32 (a thread holds one key channel of 32 columns).  Off the diagonal the
// factor of M is split at the end of its block of 32 tokens, e^(c_i - c_j) = e^(c_i - c_end) e^(c_end - c_j), both at most
// one: an exponential per row and one per token instead of one per element.  D runs under M, the next chunk's first
// products and w V run under the outputs.  Rows of a tile past the end of a portion belong to another sequence: they are
// cleared before they meet a product whose result is kept.
#include "mdb_common.cuh"

namespace mdb {

constexpr int kCtL = 128, kCtCols = 64;
constexpr int kCtWarps = 8, kCtMma = kCtWarps, kCtWeightWarps = 3, kCtThreads = (kCtWarps + 1 + kCtWeightWarps) * 32;
constexpr int kCtHalf = kCtL * 128;          // [128 rows][64 bf16]: one swizzled tile

// arrivals by warps: state and accumulators free, M, w V; by commits: G, Y1, everything; by TMA: q, k and v (per buffer); sums
// (per buffer)
enum { kCtBarOps = 0, kCtBarM, kCtBarW, kCtBarG, kCtBarY, kCtBarO, kCtBarQ, kCtBarKV, kCtBarSum = kCtBarKV + 2, kCtBars = kCtBarSum + 2 };
constexpr int kCtSums = 4 * kCtL;            // per buffer: c_j - log b_j, e^(c_end - c_j) b_j, w_j, c_i (c in log2 units)

struct CtPlan {
  static constexpr int kOffQ = 0;                              // two halves of 64 channels
  static constexpr int kOffK = kOffQ + 2 * kCtHalf;            // two buffers
  static constexpr int kOffV = kOffK + 4 * kCtHalf;            // two buffers
  static constexpr int kOffW = kOffV + 2 * kCtHalf;            // high and low parts of w V
  static constexpr int kOffS = kOffW + 2 * kCtHalf;            // high and low parts of the state [channel][64 columns]
  static constexpr int kOffStage = kOffS + 2 * kCtHalf;        // outputs on their way out, 16 rows x 128 bytes per warp
  static constexpr int kOffSums = kOffStage + kCtWarps * 2048;
  static constexpr int kOffBars = kOffSums + 2 * kCtSums * 4;
  static constexpr int kBytes = 1024 + kOffBars + 8 * kCtBars + 16;
};
static_assert(CtPlan::kBytes <= 227 * 1024, "shared memory of the chunk scan");

// tensor memory columns
constexpr uint32_t kCtG = 0, kCtMh = 128, kCtMl = 192, kCtY1 = 256 /* high | low part of S */, kCtY2 = 384, kCtD = 448;

// Four products in a row with one elected lane: left operand steps of `a_step`, right operand steps of `b_step` (descriptor
// units of 16 bytes).
__device__ __forceinline__ void umma_bf16_x4_w(uint32_t d_tmem, uint64_t a_desc, uint64_t a_step, uint64_t b_desc, uint64_t b_step, uint32_t idesc,
                                               uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, t, q;\n\t.reg .b64 a1, a2, a3, b1, b2, b3;\n\t"
      "elect.sync _|q, 0xffffffff;\n\t"
      "setp.ne.b32 p, %4, 0;\n\tsetp.eq.b32 t, 0, 0;\n\t"
      "add.u64 a1, %1, %5;\n\tadd.u64 a2, a1, %5;\n\tadd.u64 a3, a2, %5;\n\t"
      "add.u64 b1, %2, %6;\n\tadd.u64 b2, b1, %6;\n\tadd.u64 b3, b2, %6;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], a1, b1, %3, t;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], a2, b2, %3, t;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], a3, b3, %3, t;\n\t}"
      ::"r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate), "l"(a_step), "l"(b_step)
      : "memory");
}
// ... with the left operand in tensor memory: bf16 pairs, one row per lane, eight columns per step
__device__ __forceinline__ void umma_bf16_ts_x4_w(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint64_t b_step, uint32_t idesc,
                                                  uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, t, q;\n\t.reg .b64 b1, b2, b3;\n\t.reg .b32 a1, a2, a3;\n\t"
      "elect.sync _|q, 0xffffffff;\n\t"
      "setp.ne.b32 p, %4, 0;\n\tsetp.eq.b32 t, 0, 0;\n\t"
      "add.u32 a1, %1, 8;\n\tadd.u32 a2, %1, 16;\n\tadd.u32 a3, %1, 24;\n\t"
      "add.u64 b1, %2, %5;\n\tadd.u64 b2, b1, %5;\n\tadd.u64 b3, b2, %5;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [a1], b1, %3, t;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [a2], b2, %3, t;\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [a3], b3, %3, t;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(accumulate), "l"(b_step)
      : "memory");
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&v)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(taddr), "r"(v[0]), "r"(v[1]),
      "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]),
      "r"(v[14]), "r"(v[15])
      : "memory");
}
// split2 of a pair, subtracting both at once
__device__ __forceinline__ void split_pair(f32x2 xy, uint32_t& hi, uint32_t& lo) {
  const float2 v = unpack2(xy);
  hi = pack_bf16x2(v.x, v.y);
  const float2 d = unpack2(fma2(pack2(__uint_as_float(hi << 16), __uint_as_float(hi & 0xffff0000u)), pack2(-1.0f, -1.0f), xy));
  lo = pack_bf16x2(d.x, d.y);
}

// 16-byte piece c of row r of a tile with 128-byte swizzle
__device__ __forceinline__ int ct_at(int r, int c) { return r * 128 + ((c ^ (r & 7)) << 4); }

template <int NH>
__global__ void __launch_bounds__(kCtThreads, 1) chunk_scan_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                     const __grid_constant__ CUtensorMap map_v, const mdb_chunk_scan_args a) {
  using P = CtPlan;
  constexpr int DP = 64 * NH;
  extern __shared__ __align__(1024) unsigned char ct_smem_raw[];
  const uint32_t raw_base = smem_u32(ct_smem_raw);
  const uint32_t base = (raw_base + 1023u) & ~1023u;
  unsigned char* mem = ct_smem_raw + (base - raw_base);
  const uint32_t bars = base + P::kOffBars;
  volatile uint32_t* misc = reinterpret_cast<volatile uint32_t*>(mem + P::kOffBars + 8 * kCtBars);      // tensor memory base, abort flag
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z, head = blockIdx.y, col0 = blockIdx.x * kCtCols;
  const int slot = a.state_slot[seq];
  if (slot < 0) return;
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0) report_status(MDB_STATUS_BAD_SLOT);
    return;
  }
  const int t_begin = a.cu_q[seq], t_end = a.cu_q[seq + 1];
  if (t_begin >= t_end) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < kCtBars; ++s) mbar_init(bars + 8 * s, s < kCtBarW ? kCtWarps : (s == kCtBarW ? kCtWeightWarps : 1));
    misc[1] = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == kCtMma) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(const_cast<uint32_t*>(&misc[0]))), "r"(512u)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = misc[0];
  // A wait that runs out raises the abort flag; the roles then walk to the end without waiting for long again.
  auto wait = [&](int s, uint32_t parity) {
    uint32_t done;
    asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                 : "=r"(done) : "r"(bars + 8 * s), "r"(parity) : "memory");
    if (done || misc[1] != 0) return;
    if (!mbar_wait(bars + 8 * s, parity)) {
      misc[1] = 1;
      report_status(MDB_STATUS_WAIT_TIMEOUT);
    }
  };
  // chunk number c: buffer c & 1; the barriers of a buffer have parity (c >> 1) & 1, the others c & 1
  const int chunks = (t_end - t_begin + kCtL - 1) / kCtL;
  const int kvh = head / (a.heads / a.kv_heads);
  float* sums = reinterpret_cast<float*>(mem + P::kOffSums);

  if (warp == kCtMma) {
    // ---------------------------------------------------------------- products
    const uint32_t kF32 = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(128 >> 4) << 24);      // bf16 x bf16 -> fp32, M = 128
    const uint32_t id_g = kF32 | (static_cast<uint32_t>(kCtL >> 3) << 17);
    const uint32_t id_y = kF32 | (1u << 16) | (static_cast<uint32_t>(kCtCols >> 3) << 17);                     // right operand stored K first
    const uint32_t id_y1 = kF32 | (1u << 16) | (static_cast<uint32_t>(2 * kCtCols >> 3) << 17);                // both parts of S side by side
    const uint32_t id_d = id_y | (1u << 15);                                                                   // ... and the left one
    int q_loads = 0, kv_loads = 0;
    auto load_q = [&](int t0) {
      ++q_loads;
      mbar_arrive_expect_tx_w(bars + 8 * kCtBarQ, NH * kCtHalf);
#pragma unroll
      for (int h = 0; h < NH; ++h) tma_load_2d_w(base + P::kOffQ + h * kCtHalf, &map_q, kvh * DP + 64 * h, t0, bars + 8 * kCtBarQ);
    };
    auto load_kv = [&](int t0, int buf) {
      ++kv_loads;
      const uint32_t full = bars + 8 * (kCtBarKV + buf);
      mbar_arrive_expect_tx_w(full, (NH + 1) * kCtHalf);
#pragma unroll
      for (int h = 0; h < NH; ++h) tma_load_2d_w(base + P::kOffK + (2 * buf + h) * kCtHalf, &map_k, kvh * DP + 64 * h, t0, full);
      tma_load_2d_w(base + P::kOffV + buf * kCtHalf, &map_v, head * a.vdim + col0, t0, full);
    };
    // log decays and steps of four tokens per lane (past the end: no decay, no input), and their sums over the chunk
    float x[4], b[4];
    auto load_scalars = [&](int t0) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = t0 + 4 * lane + i;
        x[i] = t < t_end ? a.log_decay[t * a.ld_scalars + head] : 0.f;
        b[i] = t < t_end ? a.step[t * a.ld_scalars + head] : 0.f;
      }
    };
    auto sum_scalars = [&](int buf) {
      constexpr float kLog2e = 1.4426950408889634f;
      float c[4] = {x[0] * kLog2e, x[1] * kLog2e, x[2] * kLog2e, x[3] * kLog2e};
      c[1] += c[0]; c[2] += c[1]; c[3] += c[2];
      float s = c[3];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float p = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += p;
      }
      const float before = s - c[3], total = __shfl_sync(0xffffffffu, s, 31);
      c[0] += before; c[1] += before; c[2] += before; c[3] = s;
      const float end = __shfl_sync(0xffffffffu, s, lane | 7);      // of this block of 32 tokens
      float* at = sums + buf * kCtSums + 4 * lane;
      float w[4], m[4], f[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        w[i] = b[i] * ex2_approx(total - c[i]);
        f[i] = b[i] * ex2_approx(end - c[i]);
        m[i] = c[i] - __log2f(b[i]);                 // (step 0: +inf, weight 0)
      }
      *reinterpret_cast<float4*>(at) = make_float4(m[0], m[1], m[2], m[3]);
      *reinterpret_cast<float4*>(at + kCtL) = make_float4(f[0], f[1], f[2], f[3]);
      *reinterpret_cast<float4*>(at + 2 * kCtL) = make_float4(w[0], w[1], w[2], w[3]);
      *reinterpret_cast<float4*>(at + 3 * kCtL) = make_float4(c[0], c[1], c[2], c[3]);
      __syncwarp();
      if (lane == 0) mbar_arrive(bars + 8 * (kCtBarSum + buf));
    };
    load_q(t_begin);
    load_kv(t_begin, 0);
    load_scalars(t_begin);
    sum_scalars(0);
    const uint32_t qt = base + P::kOffQ, wt = base + P::kOffW, st = base + P::kOffS;
    for (int c = 0; c < chunks; ++c) {
      const int buf = c & 1, t0 = t_begin + c * kCtL;
      const uint32_t parity = c & 1, parity2 = (c >> 1) & 1;
      const bool more = c + 1 < chunks;
      const uint32_t kt = base + P::kOffK + buf * 2 * kCtHalf, vt = base + P::kOffV + buf * kCtHalf;
      wait(kCtBarQ, parity);
      wait(kCtBarKV + buf, parity2);
      wait(kCtBarOps, parity);
      __syncwarp();
      tc_fence_after();
      if (misc[1] != 0) break;
#pragma unroll
      for (int h = 0; h < NH; ++h)
        umma_bf16_x4_w(tmem + kCtG, umma_desc_sw128(qt + h * kCtHalf), 2, umma_desc_sw128(kt + h * kCtHalf), 2, id_g, h);
      umma_commit_w(bars + 8 * kCtBarG);
#pragma unroll
      for (int h = 0; h < NH; ++h)
        umma_bf16_x4_w(tmem + kCtY1, umma_desc_sw128(qt + h * kCtHalf), 2, umma_desc_sw128_mn(st + h * 8192), 128, id_y1, h);
      umma_commit_w(bars + 8 * kCtBarY);
      // everybody is past the chunk before this one, whose buffers these are
      if (more) {
        load_kv(t0 + kCtL, buf ^ 1);
        load_scalars(t0 + kCtL);
      }
      wait(kCtBarW, parity);
      __syncwarp();
      tc_fence_after();
#pragma unroll
      for (int i = 0; i < 4; ++i)                    // tokens 0 .. 63 and 64 .. 127, each with both parts of w V
        umma_bf16_x4_w(tmem + kCtD, umma_desc_sw128_mn(kt + (i >> 1) * 8192), 128, umma_desc_sw128_mn(wt + (i & 1) * kCtHalf + (i >> 1) * 8192), 128,
                       id_d, i);
      if (more) {
        wait(kCtBarY, parity);
        __syncwarp();
        load_q(t0 + kCtL);
      }
      wait(kCtBarM, parity);
      __syncwarp();
      tc_fence_after();
      if (misc[1] != 0) break;
#pragma unroll
      for (int i = 0; i < 4; ++i)
        umma_bf16_ts_x4_w(tmem + kCtY2, tmem + (i & 1 ? kCtMl : kCtMh) + (i >> 1) * 32, umma_desc_sw128_mn(vt + (i >> 1) * 8192), 128, id_y, i);
      umma_commit_w(bars + 8 * kCtBarO);
      if (more) sum_scalars(buf ^ 1);
    }
    if (misc[1] != 0) {                              // given up: let the copies already issued land
      mbar_wait(bars + 8 * kCtBarQ, (q_loads - 1) & 1);
      for (int n = kv_loads - 1; n >= 0 && n >= kv_loads - 2; --n) mbar_wait(bars + 8 * (kCtBarKV + (n & 1)), (n >> 1) & 1);
    }
  } else if (warp > kCtMma) {
    // -------------------------------------------------------------------- w V
    for (int c = 0; c < chunks; ++c) {
      const int buf = c & 1, t0 = t_begin + c * kCtL;
      const uint32_t parity2 = (c >> 1) & 1;
      wait(kCtBarSum + buf, parity2);
      wait(kCtBarKV + buf, parity2);
      if (c > 0) wait(kCtBarO, (c - 1) & 1);         // the last chunk's has been read
      __syncwarp();
      const float* wgt = sums + buf * kCtSums + 2 * kCtL;
      unsigned char* vt = mem + P::kOffV + buf * kCtHalf;
      // eight tokens per warp and step: four lanes per token, two of its eight 16-byte pieces each
#pragma unroll 2
      for (int j = warp - kCtMma - 1; j < kCtL / 8; j += kCtWeightWarps) {
        const int t = 8 * j + (lane >> 2);
        const float w = wgt[t];
        const f32x2 ww = pack2(w, w);
        const bool past = t0 + t >= t_end;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int at = ct_at(t, (lane & 3) + 4 * i);
          if (past) {
            const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
            *reinterpret_cast<uint4*>(vt + at) = zero;
            *reinterpret_cast<uint4*>(mem + P::kOffK + 2 * buf * kCtHalf + at) = zero;
            if (NH > 1) *reinterpret_cast<uint4*>(mem + P::kOffK + (2 * buf + 1) * kCtHalf + at) = zero;
          }
          const uint4 x = *reinterpret_cast<const uint4*>(vt + at);
          const uint32_t in[4] = {x.x, x.y, x.z, x.w};
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e)
            split_pair(mul2(pack2(__uint_as_float(in[e] << 16), __uint_as_float(in[e] & 0xffff0000u)), ww), hi[e], lo[e]);
          *reinterpret_cast<uint4*>(mem + P::kOffW + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(mem + P::kOffW + kCtHalf + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
      }
      fence_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(bars + 8 * kCtBarW);
    }
  } else {
    // ------------------------------------------------------------ everything else
    const int quad = warp & 3, hf = warp >> 2;
    const int r = 32 * quad + lane;                  // this thread's token of the chunk, and its key channel of the state
    const uint32_t lanes = static_cast<uint32_t>(32 * quad) << 16;
    const bool fresh = a.start[seq] == 0;
    const float skip = a.skip != nullptr ? a.skip[head] : 0.f;
    float* state = a.state + slot * a.state_slot_stride + static_cast<int64_t>(head) * a.vdim * DP;
    const int sc0 = col0 + 32 * hf;                  // first of this thread's 32 columns
    const bool has_state = r < DP;
    float S[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) S[i] = has_state && !fresh && sc0 + i < a.vdim ? state[static_cast<int64_t>(sc0 + i) * DP + r] : 0.f;
    auto publish = [&]() {                           // the state's two parts for the next read-out
      if (!has_state) return;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split2(S[8 * c + 2 * e], S[8 * c + 2 * e + 1], hi[e], lo[e]);
        unsigned char* at = mem + P::kOffS + ct_at(r, 4 * hf + c);
        *reinterpret_cast<uint4*>(at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(at + kCtHalf) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    };
    publish();
    auto hand_over = [&]() {                         // state and accumulators of the last chunk are done with
      fence_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bars + 8 * kCtBarOps);
    };
    hand_over();
    for (int c = 0; c < chunks; ++c) {
      const int buf = c & 1, t0 = t_begin + c * kCtL;
      const uint32_t parity = c & 1, parity2 = (c >> 1) & 1;
      const bool more = c + 1 < chunks;
      const float* cum = sums + buf * kCtSums;
      const float* blk = cum + kCtL;
      const float* crow = cum + 3 * kCtL;
      const unsigned char* vt = mem + P::kOffV + buf * kCtHalf;
      wait(kCtBarSum + buf, parity2);
      __syncwarp();
      const float ci = crow[r];
      wait(kCtBarG, parity);
      __syncwarp();
      tc_fence_after();
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int j0 = 32 * hf + 64 * half;          // 32 tokens; the warp's rows start at 32 quad
        uint32_t mh[16], ml[16];
        if (j0 > 32 * quad) {                        // behind all of them
#pragma unroll
          for (int i = 0; i < 16; ++i) mh[i] = ml[i] = 0u;
        } else {
          float g[32];
          tmem_ld32(tmem + kCtG + lanes + j0, g);
          tmem_ld_wait();
          if (j0 == 32 * quad) {                     // the diagonal: tokens up to the row's own
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              const float4 cj = *reinterpret_cast<const float4*>(cum + j0 + 4 * i);
              g[4 * i] = 4 * i <= lane ? g[4 * i] * ex2_approx(ci - cj.x) : 0.f;
              g[4 * i + 1] = 4 * i + 1 <= lane ? g[4 * i + 1] * ex2_approx(ci - cj.y) : 0.f;
              g[4 * i + 2] = 4 * i + 2 <= lane ? g[4 * i + 2] * ex2_approx(ci - cj.z) : 0.f;
              g[4 * i + 3] = 4 * i + 3 <= lane ? g[4 * i + 3] * ex2_approx(ci - cj.w) : 0.f;
            }
#pragma unroll
            for (int i = 0; i < 16; ++i) split_pair(pack2(g[2 * i], g[2 * i + 1]), mh[i], ml[i]);
          } else {
            const float e = ex2_approx(ci - crow[j0 + 31]);
            const f32x2 ee = pack2(e, e);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              f32x2 f0, f1;
              lds2(blk + j0 + 4 * i, f0, f1);
              split_pair(mul2(mul2(pack2(g[4 * i], g[4 * i + 1]), f0), ee), mh[2 * i], ml[2 * i]);
              split_pair(mul2(mul2(pack2(g[4 * i + 2], g[4 * i + 3]), f1), ee), mh[2 * i + 1], ml[2 * i + 1]);
            }
          }
        }
        tmem_st16(tmem + kCtMh + lanes + j0 / 2, mh);
        tmem_st16(tmem + kCtMl + lanes + j0 / 2, ml);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bars + 8 * kCtBarM);
      wait(kCtBarY, parity);
      wait(kCtBarKV + buf, parity2);
      __syncwarp();
      tc_fence_after();
      float y[32];
      {
        float y_lo[32];
        tmem_ld32(tmem + kCtY1 + lanes + 32 * hf, y);
        tmem_ld32(tmem + kCtY1 + lanes + kCtCols + 32 * hf, y_lo);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) y[i] += y_lo[i];
        const float e = exp2f(ci);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const uint4 x = *reinterpret_cast<const uint4*>(vt + ct_at(r, 4 * hf + c));
          const uint32_t in[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float2 f = unpack_bf16x2(in[i]);
            y[8 * c + 2 * i] = fmaf(y[8 * c + 2 * i], e, skip * f.x);
            y[8 * c + 2 * i + 1] = fmaf(y[8 * c + 2 * i + 1], e, skip * f.y);
          }
        }
      }
      const float keep = exp2f(crow[kCtL - 1]);
      wait(kCtBarO, parity);
      __syncwarp();
      tc_fence_after();
      {
        float d[32];
        tmem_ld32(tmem + kCtD + lanes + 32 * hf, d);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) S[i] = fmaf(S[i], keep, d[i]);
        if (more) {
          publish();
          hand_over();
        }
        tmem_ld32(tmem + kCtY2 + lanes + 32 * hf, d);
        tmem_ld_wait();
        // 32 rows x 128 bytes turned around in shared memory in two passes, so that whole rows leave together
        unsigned char* stage = mem + P::kOffStage + warp * 2048;
        const int piece = lane & 7, first = t0 + 32 * quad + (lane >> 3);
        const int64_t ld_out = static_cast<int64_t>(a.heads) * a.vdim;
        float* out = a.out + first * ld_out + static_cast<int64_t>(head) * a.vdim + sc0 + 4 * piece;
        const bool col_live = sc0 + 4 * piece < a.vdim;
#pragma unroll
        for (int pass = 0; pass < 2; ++pass) {
          if ((lane >> 4) == pass) {
#pragma unroll
            for (int i = 0; i < 8; ++i)
              *reinterpret_cast<float4*>(stage + ct_at(lane & 15, i)) =
                  make_float4(y[4 * i] + d[4 * i], y[4 * i + 1] + d[4 * i + 1], y[4 * i + 2] + d[4 * i + 2], y[4 * i + 3] + d[4 * i + 3]);
          }
          __syncwarp();
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float4 v = *reinterpret_cast<const float4*>(stage + ct_at(4 * i + (lane >> 3), piece));
            if (first + 16 * pass + 4 * i < t_end && col_live) *reinterpret_cast<float4*>(out + (16 * pass + 4 * i) * ld_out) = v;
          }
          __syncwarp();
        }
      }
    }
    if (has_state) {
#pragma unroll
      for (int i = 0; i < 32; ++i)
        if (sc0 + i < a.vdim) state[static_cast<int64_t>(sc0 + i) * DP + r] = S[i];
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == kCtMma) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
  }
}

template <int NH>
static int launch_chunk_scan_tc(const mdb_chunk_scan_args& a, cudaStream_t st) {
  CUtensorMap map_q, map_k, map_v;
  if (!get_tensor_map(a.q, a.m, a.kv_heads * a.dim, a.ldq, kCtL, &map_q) || !get_tensor_map(a.k, a.m, a.kv_heads * a.dim, a.ldk, kCtL, &map_k) ||
      !get_tensor_map(a.v, a.m, a.heads * a.vdim, a.ldv, kCtL, &map_v))
    return MDB_ERR_CUDA;
  static PerDeviceOnce attr_once;
  const int dev = attr_once.slot();
  if (dev < 0) return MDB_ERR_CUDA;
  if (!attr_once.done[dev]) {
    if (cudaFuncSetAttribute(chunk_scan_tc_kernel<NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, CtPlan::kBytes) != cudaSuccess) return MDB_ERR_CUDA;
    attr_once.done[dev] = true;
  }
  return mdb_launch(chunk_scan_tc_kernel<NH>, dim3((a.vdim + kCtCols - 1) / kCtCols, a.heads, a.bs), dim3(kCtThreads), CtPlan::kBytes, st, map_q, map_k,
                    map_v, a);
}

}  // namespace mdb
