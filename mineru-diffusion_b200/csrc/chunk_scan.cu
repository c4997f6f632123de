// The decay scan S <- a S + b k v^T, o = S^T q + skip v over prompt portions in chunks of 64 tokens on the tensor cores.
// With c_i the sum of the log decays of a chunk's tokens up to i,
//   o_i = e^(c_i) S^T q_i + sum_(j <= i) (q_i . k_j) e^(c_i - c_j) b_j v_j + skip v_i,
//   S  <- e^(c_last) S + sum_j e^(c_last - c_j) b_j k_j v_j^T,
// four matrix products per chunk.  q, k and v are bf16 (the activations behind a projection); the state stays in fp32
// accumulators from the first chunk of a portion to the last, and everything else that enters a product -- the state in the
// read-out, the weighted scores, the weighted keys -- enters as the sum of two bf16 numbers, 16 significant bits.
//
// A CTA owns PB value columns of one head of one sequence.  Eight warps: for the outputs four groups of 16 tokens times
// two halves of the columns, for the state blocks of 16 key channels times half the columns.  Two barriers per chunk; the
// next chunk's operands are requested (cp.async) as soon as q has been read.
#include "mdb_common.cuh"

namespace mdb {

constexpr int kChunk = 64, kChunkThreads = 256;

template <int DP, int PB>
struct ChunkPlan {
  static constexpr int kQS = DP + 8, kVS = PB + 8;                      // row strides in bf16; the pads spread rows over the banks
  static constexpr int kTileK = kChunk * kQS * 2, kTileV = kChunk * kVS * 2, kTileS = DP * kVS * 2;
  static constexpr int kOffQ = 0;
  static constexpr int kOffK = kOffQ + kTileK;                          // two buffers
  static constexpr int kOffV = kOffK + 2 * kTileK;                      // two buffers
  static constexpr int kOffS = kOffV + 2 * kTileV;                      // high and low parts of the state, [DP][kVS]
  static constexpr int kOffRaw = kOffS + 2 * kTileS;                    // two buffers of log decays and steps
  static constexpr int kOffCum = kOffRaw + 2 * 2 * kChunk * 4;          // c_j - log b_j in log2 units, the state's weights, c_i
  static constexpr int kBytes = kOffCum + 3 * kChunk * 4;
};

// high and low bf16 parts of two numbers
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}

template <int DP, int PB>
__global__ void __launch_bounds__(kChunkThreads, DP <= 128 ? 2 : 1) chunk_scan_kernel(const mdb_chunk_scan_args a) {
  using P = ChunkPlan<DP, PB>;
  constexpr int HC = PB / 2, NT = HC / 8;          // columns of a half, and their tiles
  constexpr int NU = DP / 64;                      // state blocks (16 channels x HC columns) of a warp
  extern __shared__ __align__(16) unsigned char chunk_smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z, head = blockIdx.y, col0 = blockIdx.x * PB;
  const int slot = a.state_slot[seq];
  if (slot < 0) return;
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0) report_status(MDB_STATUS_BAD_SLOT);
    return;
  }
  const int t_begin = a.cu_q[seq], t_end = a.cu_q[seq + 1];
  if (t_begin >= t_end) return;
  const bool fresh = a.start[seq] == 0;
  const int kvh = head / (a.heads / a.kv_heads);
  const float skip = a.skip != nullptr ? a.skip[head] : 0.f;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j2 = 2 * (lane & 3);
  const int rg = warp & 3, ch = warp >> 2;         // outputs: tokens 16 rg .. of the chunk, column half ch
  const uint32_t base = smem_u32(chunk_smem);
  float* cum = reinterpret_cast<float*>(chunk_smem + P::kOffCum);
  float* wgt = cum + kChunk;
  float* crow = wgt + kChunk;

  const bf16* q = static_cast<const bf16*>(a.q) + static_cast<int64_t>(kvh) * a.dim;
  const bf16* k = static_cast<const bf16*>(a.k) + static_cast<int64_t>(kvh) * a.dim;
  const bf16* v = static_cast<const bf16*>(a.v) + static_cast<int64_t>(head) * a.vdim + col0;
  auto copy16 = [&](uint32_t dst, const bf16* src, bool live) {       // size 0 reads nothing and writes zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
  };
  auto request = [&](int t0, int buf) {
    const int n = t_end - t0;
    if (n > 0) {
      for (int i = threadIdx.x; i < kChunk * (DP / 8); i += kChunkThreads) {
        const int t = i / (DP / 8), c = i % (DP / 8) * 8;
        const bool live = t < n && c < a.dim;
        const int64_t row = live ? t0 + t : t_begin;
        copy16(base + P::kOffQ + (t * P::kQS + c) * 2, q + row * a.ldq + (live ? c : 0), live);
        copy16(base + P::kOffK + buf * P::kTileK + (t * P::kQS + c) * 2, k + row * a.ldk + (live ? c : 0), live);
      }
      for (int i = threadIdx.x; i < kChunk * (PB / 8); i += kChunkThreads) {
        const int t = i / (PB / 8), c = i % (PB / 8) * 8;
        const bool live = t < n && col0 + c < a.vdim;
        copy16(base + P::kOffV + buf * P::kTileV + (t * P::kVS + c) * 2, v + (live ? (t0 + t) * a.ldv + c : 0), live);
      }
      if (threadIdx.x < 2 * kChunk) {              // tokens past the end: no decay, no input
        const int t = threadIdx.x & (kChunk - 1);
        const float* src = threadIdx.x < kChunk ? a.log_decay : a.step;
        const bool live = t < n;
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(base + P::kOffRaw + (buf * 2 * kChunk + threadIdx.x) * 4),
                     "l"(src + (live ? (t0 + t) * a.ld_scalars + head : 0)), "r"(live ? 4 : 0) : "memory");
      }
    }
    cp_async_commit();
  };
  request(t_begin, 0);

  // the state: unit u = 16 channels (u >> 1) x column half (u & 1); a thread holds the accumulator fragments
  float st[NU][NT][4];
  float* state = a.state + slot * a.state_slot_stride + static_cast<int64_t>(head) * a.vdim * DP;
#pragma unroll
  for (int i = 0; i < NU; ++i) {
    const int u = warp * NU + i;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = 16 * (u >> 1) + g + 8 * (e >> 1), col = col0 + (u & 1) * HC + 8 * n + j2 + (e & 1);
        st[i][n][e] = !fresh && col < a.vdim ? state[static_cast<int64_t>(col) * DP + row] : 0.f;
      }
  }
  auto publish = [&]() {                           // the state's two parts for the read-out
#pragma unroll
    for (int i = 0; i < NU; ++i) {
      const int u = warp * NU + i;
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t hi, lo;
          split2(st[i][n][2 * r], st[i][n][2 * r + 1], hi, lo);
          const int at = ((16 * (u >> 1) + g + 8 * r) * P::kVS + (u & 1) * HC + 8 * n + j2) * 2;
          *reinterpret_cast<uint32_t*>(chunk_smem + P::kOffS + at) = hi;
          *reinterpret_cast<uint32_t*>(chunk_smem + P::kOffS + P::kTileS + at) = lo;
        }
    }
  };
  publish();

  // per-lane offsets of the operand loads
  const uint32_t a_off = ((lane & 15) * P::kQS + (lane >> 4) * 8) * 2;                                        // rows x columns
  const uint32_t k_off = (((lane & 7) + ((lane >> 4) & 1) * 8) * P::kQS + ((lane >> 3) & 1) * 8) * 2;         // rows are the output's columns
  const uint32_t v_off = (((lane & 7) + ((lane >> 3) & 1) * 8) * P::kVS + (lane >> 4) * 8) * 2;               // transposed
  const uint32_t kt_off = (((lane & 7) + ((lane >> 4) & 1) * 8) * P::kQS + ((lane >> 3) & 1) * 8) * 2;        // transposed, as left operand
  int buf = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += kChunk, buf ^= 1) {
    cp_async_wait<0>();
    __syncthreads();                               // the chunk has landed, the state's parts are written
    if (warp == 0) {
      const float* raw = reinterpret_cast<const float*>(chunk_smem + P::kOffRaw) + buf * 2 * kChunk;
      // inclusive sums over 64 tokens, two per lane
      const float x0 = raw[2 * lane] * 1.4426950408889634f, x1 = raw[2 * lane + 1] * 1.4426950408889634f;
      float s = x0 + x1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float p = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += p;
      }
      const float total = __shfl_sync(0xffffffffu, s, 31), b0 = raw[kChunk + 2 * lane], b1 = raw[kChunk + 2 * lane + 1];
      const float c0 = s - x1, c1 = s;
      *reinterpret_cast<float2*>(crow + 2 * lane) = make_float2(c0, c1);
      *reinterpret_cast<float2*>(cum + 2 * lane) = make_float2(c0 - log2f(b0), c1 - log2f(b1));      // (step 0: +inf, weight 0)
      *reinterpret_cast<float2*>(wgt + 2 * lane) = make_float2(b0 * exp2f(total - c0), b1 * exp2f(total - c1));
    }
    const uint32_t qt = base + P::kOffQ + 16 * rg * P::kQS * 2, kt = base + P::kOffK + buf * P::kTileK, vt = base + P::kOffV + buf * P::kTileV;
    const uint32_t sh = base + P::kOffS + ch * HC * 2;
    float G[8][4], Y[NT][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) G[i][0] = G[i][1] = G[i][2] = G[i][3] = 0.f;
#pragma unroll
    for (int i = 0; i < NT; ++i) Y[i][0] = Y[i][1] = Y[i][2] = Y[i][3] = 0.f;
#pragma unroll 4
    for (int ks = 0; ks < DP / 16; ++ks) {
      uint32_t qf[4];
      ldsm4(qt + a_off + 32 * ks, qf);
#pragma unroll
      for (int p = 0; p < NT / 2; ++p) {
        uint32_t h[4], l[4];
        const uint32_t at = sh + v_off + (16 * ks * P::kVS + 16 * p) * 2;
        ldsm4_t(at, h);
        ldsm4_t(at + P::kTileS, l);
        mma16816(Y[2 * p], qf, h[0], h[1]);
        mma16816(Y[2 * p + 1], qf, h[2], h[3]);
        mma16816(Y[2 * p], qf, l[0], l[1]);
        mma16816(Y[2 * p + 1], qf, l[2], l[3]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (j > rg) break;
        uint32_t b[4];
        ldsm4(kt + k_off + (16 * j * P::kQS + 16 * ks) * 2, b);
        mma16816(G[2 * j], qf, b[0], b[1]);
        mma16816(G[2 * j + 1], qf, b[2], b[3]);
      }
    }
    __syncthreads();                               // q and the state's parts have been read; sums and weights are written
    request(t0 + kChunk, buf ^ 1);
    const int r0 = 16 * rg + g;
    const float c0 = crow[r0], c1 = crow[r0 + 8];
    {
      const float e0 = exp2f(c0), e1 = exp2f(c1);
#pragma unroll
      for (int i = 0; i < NT; ++i) { Y[i][0] *= e0; Y[i][1] *= e0; Y[i][2] *= e1; Y[i][3] *= e1; }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (j > rg) break;
      uint32_t mh[4], ml[4];
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int t = 16 * j + 8 * n + j2;
        const float2 cj = *reinterpret_cast<const float2*>(cum + t);
        const float (&x)[4] = G[2 * j + n];
        float m0 = x[0] * ex2_approx(c0 - cj.x), m1 = x[1] * ex2_approx(c0 - cj.y);
        float m2 = x[2] * ex2_approx(c1 - cj.x), m3 = x[3] * ex2_approx(c1 - cj.y);
        if (j == rg) {                             // the diagonal tile: tokens up to the row's own
          m0 = t <= r0 ? m0 : 0.f;
          m1 = t + 1 <= r0 ? m1 : 0.f;
          m2 = t <= r0 + 8 ? m2 : 0.f;
          m3 = t + 1 <= r0 + 8 ? m3 : 0.f;
        }
        split2(m0, m1, mh[2 * n], ml[2 * n]);
        split2(m2, m3, mh[2 * n + 1], ml[2 * n + 1]);
      }
#pragma unroll
      for (int p = 0; p < NT / 2; ++p) {
        uint32_t b[4];
        ldsm4_t(vt + v_off + (16 * j * P::kVS + ch * HC + 16 * p) * 2, b);
        mma16816(Y[2 * p], mh, b[0], b[1]);
        mma16816(Y[2 * p + 1], mh, b[2], b[3]);
        mma16816(Y[2 * p], ml, b[0], b[1]);
        mma16816(Y[2 * p + 1], ml, b[2], b[3]);
      }
    }
    // outputs of the 16 tokens
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = r0 + 8 * r;
      if (t0 + t >= t_end) continue;
      float* out = a.out + (static_cast<int64_t>(t0 + t) * a.heads + head) * a.vdim + col0;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int c = ch * HC + 8 * n + j2;
        if (col0 + c >= a.vdim) continue;          // (an even number of columns)
        const float2 vv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(chunk_smem + P::kOffV + buf * P::kTileV + (t * P::kVS + c) * 2));
        *reinterpret_cast<float2*>(out + c) = make_float2(fmaf(skip, vv.x, Y[n][2 * r]), fmaf(skip, vv.y, Y[n][2 * r + 1]));
      }
    }
    // the state
    const float total = exp2f(crow[kChunk - 1]);
#pragma unroll
    for (int i = 0; i < NU; ++i)
#pragma unroll
      for (int n = 0; n < NT; ++n) { st[i][n][0] *= total; st[i][n][1] *= total; st[i][n][2] *= total; st[i][n][3] *= total; }
#pragma unroll
    for (int ks = 0; ks < kChunk / 16; ++ks) {
      const float2 w0 = *reinterpret_cast<const float2*>(wgt + 16 * ks + j2), w1 = *reinterpret_cast<const float2*>(wgt + 16 * ks + 8 + j2);
      uint32_t kh[4], kl[4];
#pragma unroll
      for (int i = 0; i < NU; ++i) {
        const int u = warp * NU + i;
        if (NU % 2 != 0 || i % 2 == 0) {           // (an even unit and the one behind it share their channels)
          uint32_t kf[4];
          ldsm4_t(kt + kt_off + (16 * ks * P::kQS + 16 * (u >> 1)) * 2, kf);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 x = unpack_bf16x2(kf[e]), w = e < 2 ? w0 : w1;
            split2(x.x * w.x, x.y * w.y, kh[e], kl[e]);
          }
        }
#pragma unroll
        for (int p = 0; p < NT / 2; ++p) {
          uint32_t b[4];
          ldsm4_t(vt + v_off + (16 * ks * P::kVS + (u & 1) * HC + 16 * p) * 2, b);
          mma16816(st[i][2 * p], kh, b[0], b[1]);
          mma16816(st[i][2 * p + 1], kh, b[2], b[3]);
          mma16816(st[i][2 * p], kl, b[0], b[1]);
          mma16816(st[i][2 * p + 1], kl, b[2], b[3]);
        }
      }
    }
    publish();
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < NU; ++i) {
    const int u = warp * NU + i;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = 16 * (u >> 1) + g + 8 * (e >> 1), col = col0 + (u & 1) * HC + 8 * n + j2 + (e & 1);
        if (col < a.vdim) state[static_cast<int64_t>(col) * DP + row] = st[i][n][e];
      }
  }
}

template <int DP, int PB>
static int launch_chunk_scan(const mdb_chunk_scan_args& a, cudaStream_t st) {
  constexpr int smem = ChunkPlan<DP, PB>::kBytes;
  static_assert(smem <= 227 * 1024, "shared memory of the chunk scan");
  static PerDeviceOnce attr_once;
  const int dev = attr_once.slot();
  if (dev < 0) return MDB_ERR_CUDA;
  if (!attr_once.done[dev]) {
    if (cudaFuncSetAttribute(chunk_scan_kernel<DP, PB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return MDB_ERR_CUDA;
    attr_once.done[dev] = true;
  }
  return mdb_launch(chunk_scan_kernel<DP, PB>, dim3((a.vdim + PB - 1) / PB, a.heads, a.bs), dim3(kChunkThreads), smem, st, a);
}

template <int DP>
static int launch_chunk_scan_cols(const mdb_chunk_scan_args& a, cudaStream_t st) {
  // narrow column blocks where wide ones would leave SMs idle
  const int64_t wide = static_cast<int64_t>((a.vdim + 63) / 64) * a.heads * a.bs;
  return a.vdim <= 32 || wide < 148 ? launch_chunk_scan<DP, 32>(a, st) : launch_chunk_scan<DP, 64>(a, st);
}

// the form for portions of more than one chunk (defined with the tensor-memory kernels' helpers in scope)
template <int NH> static int launch_chunk_scan_tc(const mdb_chunk_scan_args& a, cudaStream_t st);

}  // namespace mdb

using namespace mdb;

extern "C" {

int mdb_chunk_scan_supported(int dim_pad, int vdim) {
  return (dim_pad == 64 || dim_pad == 128 || dim_pad == 192 || dim_pad == 256) && vdim % 8 == 0 ? 1 : 0;
}

int mdb_chunk_scan(const mdb_chunk_scan_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_chunk_scan_args a = *args;
  MDB_REQUIRE(a.bs >= 0 && a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.vdim > 0, MDB_ERR_ARG);
  if (a.bs == 0) return MDB_OK;
  MDB_REQUIRE(a.q && a.k && a.v && a.log_decay && a.step && a.state && a.cu_q && a.start && a.state_slot && a.out, MDB_ERR_ARG);
  MDB_REQUIRE(a.m > 0 && a.dim > 0 && a.dim <= a.dim_pad && a.ldq >= static_cast<int64_t>(a.kv_heads) * a.dim && a.ldk >= static_cast<int64_t>(a.kv_heads) * a.dim &&
                  a.ldv >= static_cast<int64_t>(a.heads) * a.vdim && a.ld_scalars >= 0,
              MDB_ERR_ARG);
  MDB_REQUIRE(a.dim % 8 == 0 && a.ldq % 8 == 0 && a.ldk % 8 == 0 && a.ldv % 8 == 0 && mdb_aligned16(a.q) && mdb_aligned16(a.k) &&
                  mdb_aligned16(a.v) && mdb_aligned16(a.out),
              MDB_ERR_ALIGN);
  MDB_REQUIRE(mdb_chunk_scan_supported(a.dim_pad, a.vdim) && a.heads <= 65535 && a.bs <= 65535, MDB_ERR_UNSUPPORTED);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool long_chunks = a.max_q > kChunk && a.dim == a.dim_pad;
  switch (a.dim_pad) {
    case 64: return long_chunks ? launch_chunk_scan_tc<1>(a, st) : launch_chunk_scan_cols<64>(a, st);
    case 128: return long_chunks ? launch_chunk_scan_tc<2>(a, st) : launch_chunk_scan_cols<128>(a, st);
    case 192: return launch_chunk_scan_cols<192>(a, st);
    default: return launch_chunk_scan_cols<256>(a, st);
  }
}

}  // extern "C"
