// Recurrent mixers with a matrix state per head: the gated delta rule with one decay per key channel, and the mLSTM
// matrix memory.  One scan kernel serves prompts, portions of prompts and decoding; the state lives in fp32 in a slot
// per sequence and every product of the recurrence is an fp32 FMA (packed two at a time, fma.rn.f32x2).
//
// State layout: [slot][head][value column][key channel padded to a multiple of 32], so a value column is contiguous.
// The columns of a head are independent of one another (the delta rule's correction of a column only needs that
// column), so a CTA owns a block of columns: eight lanes share a column, each holding every eighth float4 of it in
// registers, CPT columns per thread; a token needs one three-step shuffle reduction over the eight lanes.  k, q and
// the decays of a block of tokens come through a double-buffered shared-memory stage (cp.async).
//
// The read-out of the delta rule is rewritten so that both products with the old state share one reduction:
//   a = (g S)^T k,  b = (g S)^T q,  u = beta (v - a),  o = b + (k . q) u,  S <- g S + k u^T.
#include "mdb_common.cuh"

namespace mdb {

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ void lds2(uint32_t addr, f32x2& a, f32x2& b) {
  asm volatile("ld.shared.v2.u64 {%0, %1}, [%2];" : "=l"(a), "=l"(b) : "r"(addr));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float sum8(float v) {
  v += __shfl_xor_sync(0xffffffffu, v, 4);
  v += __shfl_xor_sync(0xffffffffu, v, 2);
  v += __shfl_xor_sync(0xffffffffu, v, 1);
  return v;
}

// ---------------------------------------------------------------------------
// Before the delta scan: short convolution + silu of q, k and v, unit norm of q and k, k . q, sigmoid of beta.
// Units of a row, one warp each: kv_heads (q and k of one head), heads (v of one head), one for beta, and, where the
// projection came as split-k slices, the copy of its low-rank columns for the GEMM that follows.
// ---------------------------------------------------------------------------
constexpr int kPrepWarps = 4;
constexpr int kMaxTaps = 16;

template <typename T>
struct ConvCtx {
  const mdb_delta_prep_args* a;
  int64_t row;
  int tloc, slot;      // token index inside this step's portion; state slot (-1: starts from zeros)
  // input of channel `col` of projection `src`, `back` tokens ago
  __device__ __forceinline__ float at(const mdb_rows& src, int col, int channel, int back) const {
    if (back <= tloc) return rows_at<T>(src, row - back, col);
    const int idx = a->taps - 1 - (back - tloc);
    if (slot < 0 || idx < 0) return 0.f;
    return act_to_f(static_cast<const T*>(a->conv_state)[slot * a->conv_slot_stride + static_cast<int64_t>(idx) * a->channels + channel]);
  }
  __device__ __forceinline__ float conv_silu(const mdb_rows& src, const float* w, int col, int channel) const {
    float acc = 0.f;
    for (int j = 0; j < a->taps; ++j) acc = fmaf(w[static_cast<int64_t>(col) * a->taps + j], at(src, col, channel, a->taps - 1 - j), acc);
    return acc / (1.0f + expf(-acc));
  }
};

template <typename T>
__global__ void __launch_bounds__(kPrepWarps * 32) delta_prep_kernel(const mdb_delta_prep_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.y * kPrepWarps + (threadIdx.x >> 5);
  const int seq = a.row_seq[row];
  const int slot = a.state_slot[seq];
  if (slot < 0) return;
  if (slot >= a.num_slots) {
    if (lane == 0) report_status(MDB_STATUS_BAD_SLOT);
    return;
  }
  ConvCtx<T> cx = {&a, row, static_cast<int>(row) - a.cu_q[seq], a.start[seq] == 0 ? -1 : slot};
  // one-token portions move the convolution state along right here: the warp owns its channels
  auto shift = [&](const mdb_rows& src, int col, int channel) {
    if (!a.shift_state || a.taps < 2) return;
    T* st = static_cast<T*>(a.conv_state) + slot * a.conv_slot_stride + channel;
    float keep[kMaxTaps];
#pragma unroll 1
    for (int j = 0; j < a.taps - 1; ++j) keep[j] = cx.at(src, col, channel, a.taps - 2 - j);
#pragma unroll 1
    for (int j = 0; j < a.taps - 1; ++j) st[static_cast<int64_t>(j) * a.channels] = act_from_f<T>(keep[j]);
  };
  if (unit < a.kv_heads) {
    float* qo = a.q_out + (row * a.kv_heads + unit) * a.dim_pad;
    float* ko = a.k_out + (row * a.kv_heads + unit) * a.dim_pad;
    const int kq_channels = a.kv_heads * a.dim;
    float sq = 0.f, sk = 0.f, dot = 0.f;
    for (int d = lane; d < a.dim_pad; d += 32) {
      float q = 0.f, k = 0.f;
      if (d < a.dim) {
        const int col = unit * a.dim + d;
        q = cx.conv_silu(a.q, a.conv_q, col, col);
        k = cx.conv_silu(a.k, a.conv_k, col, kq_channels + col);
        shift(a.q, col, col);
        shift(a.k, col, kq_channels + col);
      }
      qo[d] = q;
      ko[d] = k;
      sq += q * q;
      sk += k * k;
    }
    const float rq = (1.0f / sqrtf(warp_sum(sq) + 1e-6f)) * (1.0f / sqrtf(static_cast<float>(a.dim)));
    const float rk = 1.0f / sqrtf(warp_sum(sk) + 1e-6f);
    for (int d = lane; d < a.dim_pad; d += 32) {       // a lane re-reads what it wrote itself
      const float q = qo[d] * rq, k = ko[d] * rk;
      qo[d] = q;
      ko[d] = k;
      dot += q * k;
    }
    dot = warp_sum(dot);
    if (lane == 0) a.kq_out[row * a.kv_heads + unit] = dot;
    return;
  }
  const int vu = unit - a.kv_heads;
  if (vu < a.heads) {
    float* vo = a.v_out + (row * a.heads + vu) * a.vdim;
    for (int d = lane; d < a.vdim; d += 32) {
      const int col = vu * a.vdim + d, channel = 2 * a.kv_heads * a.dim + col;
      const float v = cx.conv_silu(a.v, a.conv_v, col, channel);
      shift(a.v, col, channel);
      vo[d] = v;
    }
    return;
  }
  if (vu == a.heads) {
    for (int h = lane; h < a.heads; h += 32) a.beta_out[row * a.heads + h] = sigmoid_f(rows_at<T>(a.b, row, h));
    return;
  }
  const int cu = vu - a.heads - 1;       // copy unit: 128 columns
  if (a.copy_cols > 0 && cu * 128 < a.copy_cols) {
    const int c = cu * 128 + lane * 4;
    if (c < a.copy_cols) act_store4(static_cast<T*>(a.copy_out) + row * a.copy_ld + c, rows_at4<T>(a.copy, row, c));
  }
}

// The last taps - 1 inputs of every channel after a step of arbitrary portions: one thread per (sequence, channel).
template <typename T>
__global__ void __launch_bounds__(256) conv_state_kernel(const mdb_delta_prep_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.y;
  const int channel = blockIdx.x * 256 + threadIdx.x;
  const int slot = a.state_slot[seq];
  if (slot < 0 || slot >= a.num_slots || channel >= a.channels) return;
  const int t0 = a.cu_q[seq], n = a.cu_q[seq + 1] - t0;
  if (n <= 0) return;
  const int kc = a.kv_heads * a.dim;
  const mdb_rows& src = channel < kc ? a.q : (channel < 2 * kc ? a.k : a.v);
  const int col = channel < kc ? channel : (channel < 2 * kc ? channel - kc : channel - 2 * kc);
  ConvCtx<T> cx = {&a, t0 + n - 1, n - 1, a.start[seq] == 0 ? -1 : slot};
  float keep[kMaxTaps];
#pragma unroll 1
  for (int j = 0; j < a.taps - 1; ++j) keep[j] = cx.at(src, col, channel, a.taps - 2 - j);
  T* st = static_cast<T*>(a.conv_state) + slot * a.conv_slot_stride + channel;
#pragma unroll 1
  for (int j = 0; j < a.taps - 1; ++j) st[static_cast<int64_t>(j) * a.channels] = act_from_f<T>(keep[j]);
}

// g = exp(-exp(A_log) * softplus(x + dt_bias)), laid out [row][head][dim_pad] (padding channels: 1)
__global__ void __launch_bounds__(256) channel_decay_kernel(const float* x, int64_t ldx,
                                                            const float* a_log, const float* dt_bias,
                                                            float* g, int64_t total, int heads, int dim, int dim_pad) {
  pdl_launch_dependents();
  pdl_wait();
  for (int64_t i = blockIdx.x * static_cast<int64_t>(256) + threadIdx.x; i < total; i += static_cast<int64_t>(gridDim.x) * 256) {
    const int d = static_cast<int>(i % dim_pad);
    const int64_t rh = i / dim_pad;
    const int h = static_cast<int>(rh % heads);
    float r = 1.f;
    if (d < dim) r = expf(-expf(a_log[h]) * softplus_f(x[(rh / heads) * ldx + h * dim + d] + dt_bias[h * dim + d]));
    g[i] = r;
  }
}

// Before the mLSTM scan: q scaled, k, v as fp32 rows (key channels padded with zeros), and the two log gates.
template <typename T>
__global__ void __launch_bounds__(128) mlstm_prep_kernel(const mdb_mlstm_prep_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int nq = a.heads * a.dim_pad, nv = a.heads * a.vdim;
  const float scale = 1.0f / sqrtf(static_cast<float>(a.dim));
  for (int i = blockIdx.y * 128 + threadIdx.x; i < nq + nv + a.heads; i += gridDim.y * 128) {
    if (i < nq) {
      const int h = i / a.dim_pad, d = i % a.dim_pad;
      float q = 0.f, k = 0.f;
      if (d < a.dim) {
        q = rows_at<T>(a.q, row, h * a.dim + d) * scale;
        k = rows_at<T>(a.k, row, h * a.dim + d);
      }
      a.q_out[row * nq + i] = q;
      a.k_out[row * nq + i] = k;
    } else if (i < nq + nv) {
      a.v_out[row * nv + (i - nq)] = rows_at<T>(a.v, row, i - nq);
    } else {
      const int h = i - nq - nv;
      const float zi = rows_at<T>(a.i, row, h) + a.bias_i[h], zf = rows_at<T>(a.f, row, h) + a.bias_f[h];
      a.log_i[row * a.heads + h] = a.cap * tanhf(zi / a.cap);
      a.log_f[row * a.heads + h] = -softplus_f(-(a.cap * tanhf(zf / a.cap)));
    }
  }
}

// ---------------------------------------------------------------------------
// The scan
// ---------------------------------------------------------------------------
enum { kScanDelta = MDB_SCAN_DELTA, kScanMlstm = MDB_SCAN_MLSTM };
constexpr int kScanFusedThreads = 512, kScanFusedMaxDim = 256;
constexpr int kScanBlockCols = 32;       // granularity of the copies of the mLSTM normaliser

// floats of one stage: k, q (and the decays) of tb tokens, their values for `cols` columns, two scalars per token
__host__ __device__ constexpr int scan_stage_floats(int mode, int dp, int tb, int cols) {
  return tb * ((mode == kScanDelta ? 3 : 2) * dp + cols + 4);
}

// FUSED: every sequence brings one token and the CTA owns all columns of the head; the decay is computed from the raw
// projection and the head's output is normalised, gated and stored as the next projection's input.
template <typename T, int MODE, int NCH, int CPT, int TB, bool FUSED>
__global__ void __launch_bounds__(FUSED ? kScanFusedThreads : 256) scan_kernel(const mdb_scan_args a, const int cols) {
  constexpr int DP = NCH * 32;
  extern __shared__ __align__(16) float scan_smem[];
  __shared__ float sh_gate[3 * TB];      // mLSTM: forget factor, input factor, exp(-m) per token of the block
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z, head = blockIdx.y;
  const int l8 = threadIdx.x & 7, cg = threadIdx.x >> 3;
  const int col0 = blockIdx.x * cols, mycol = col0 + cg * CPT;
  const int slot = a.state_slot[seq];
  if (slot < 0) return;
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0) report_status(MDB_STATUS_BAD_SLOT);
    return;
  }
  const int t_begin = a.cu_q[seq], t_end = a.cu_q[seq + 1];
  if (t_end <= t_begin) return;
  const bool fresh = a.start[seq] == 0;
  const int kvh = head / (a.heads / a.kv_heads);
  float* state = a.state + slot * a.state_slot_stride + static_cast<int64_t>(head) * a.vdim * DP;

  f32x2 S[CPT][NCH * 2];
#pragma unroll
  for (int i = 0; i < CPT; ++i)
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && mycol + i < a.vdim)
        v = *reinterpret_cast<const float4*>(state + static_cast<int64_t>(mycol + i) * DP + c * 32 + l8 * 4);
      S[i][2 * c] = pack2(v.x, v.y);
      S[i][2 * c + 1] = pack2(v.z, v.w);
    }
  // mLSTM: the normaliser n and the running maximum m.  Each block of 32 columns keeps a copy of both, so that CTAs of
  // one head never read what another writes.
  f32x2 N[MODE == kScanMlstm ? NCH * 2 : 1];
  float run_max = 0.f;
  const int blocks = (a.vdim + kScanBlockCols - 1) / kScanBlockCols;
  float* nstate = nullptr;
  float* mstate = nullptr;
  if (MODE == kScanMlstm) {
    const int64_t hb = (static_cast<int64_t>(slot) * a.heads + head) * blocks;
    nstate = a.nstate + hb * DP;
    mstate = a.mstate + hb;
    const int b0 = col0 / kScanBlockCols;
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh) v = *reinterpret_cast<const float4*>(nstate + static_cast<int64_t>(b0) * DP + c * 32 + l8 * 4);
      N[2 * c] = pack2(v.x, v.y);
      N[2 * c + 1] = pack2(v.z, v.w);
    }
    if (!fresh) run_max = mstate[b0];
  }

  const uint32_t smem0 = smem_u32(scan_smem);
  const int stage_floats = scan_stage_floats(MODE, DP, TB, cols);
  constexpr int kVec = MODE == kScanDelta ? 3 : 2;
  const int off_v = TB * kVec * DP, off_s = off_v + TB * cols;
  auto stage = [&](int t0, int buf) {
    const int n = min(TB, t_end - t0);
    const uint32_t base = smem0 + buf * stage_floats * 4;
    for (int i = threadIdx.x; i < n * (DP / 4); i += blockDim.x) {
      const int t = i / (DP / 4), c = i % (DP / 4);
      const int64_t krow = (static_cast<int64_t>(t0 + t) * a.kv_heads + kvh) * DP + c * 4;
      cp_async16(base + (t * DP + c * 4) * 4, a.k + krow);
      cp_async16(base + ((TB + t) * DP + c * 4) * 4, a.q + krow);
      if (MODE == kScanDelta && !FUSED)
        cp_async16(base + ((2 * TB + t) * DP + c * 4) * 4, a.g + (static_cast<int64_t>(t0 + t) * a.heads + head) * DP + c * 4);
    }
    if (MODE == kScanDelta && FUSED) {
      for (int i = threadIdx.x; i < n * DP; i += blockDim.x) {
        const int t = i / DP, d = i % DP;
        float r = 1.f;
        if (d < a.dim)
          r = expf(-expf(a.a_log[head]) * softplus_f(rows_at<float>(a.raw_decay, t0 + t, head * a.dim + d) + a.dt_bias[head * a.dim + d]));
        scan_smem[buf * stage_floats + (2 * TB + t) * DP + d] = r;
      }
    }
    for (int i = threadIdx.x; i < n * cols; i += blockDim.x) {
      const int t = i / cols, c = i % cols;
      if (col0 + c < a.vdim)
        cp_async4(base + (off_v + t * cols + c) * 4, a.v + (static_cast<int64_t>(t0 + t) * a.heads + head) * a.vdim + col0 + c);
      else
        scan_smem[buf * stage_floats + off_v + t * cols + c] = 0.f;
    }
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
      const int64_t t = t0 + i;
      cp_async4(base + (off_s + 2 * i) * 4, a.s0 + t * a.heads + head);
      cp_async4(base + (off_s + 2 * i + 1) * 4, MODE == kScanDelta ? a.s1 + t * a.kv_heads + kvh : a.s1 + t * a.heads + head);
    }
    cp_async_commit();
  };

  float out[CPT];
  stage(t_begin, 0);
  int buf = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += TB, buf ^= 1) {
    const int n = min(TB, t_end - t0);
    if (t0 + TB < t_end) {
      stage(t0 + TB, buf ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const float* st = scan_smem + buf * stage_floats;
    const uint32_t st_addr = smem0 + buf * stage_floats * 4;
    if (MODE == kScanMlstm) {
      // m_t = max(f_t + m_(t-1), i_t) over the block as a scan of the maps x -> max(x + F, I)
      if (threadIdx.x < 32) {
        const int l = threadIdx.x;
        const float li = l < n ? st[off_s + 2 * l] : -INFINITY, lf = l < n ? st[off_s + 2 * l + 1] : 0.f;
        float F = lf, I = li;
#pragma unroll
        for (int o = 1; o < TB; o <<= 1) {
          const float Fp = __shfl_up_sync(0xffffffffu, F, o), Ip = __shfl_up_sync(0xffffffffu, I, o);
          if (l >= o) { I = fmaxf(Ip + F, I); F += Fp; }
        }
        const float m = fmaxf(F + run_max, I);
        float mp = __shfl_up_sync(0xffffffffu, m, 1);
        if (l == 0) mp = run_max;
        if (l < n) {
          sh_gate[l] = expf(lf + mp - m);
          sh_gate[TB + l] = expf(li - m);
          sh_gate[2 * TB + l] = expf(-m);
        }
        run_max = __shfl_sync(0xffffffffu, m, n - 1);
      }
      __syncthreads();
    }
    for (int t = 0; t < n; ++t) {
      const uint32_t ka = st_addr + (t * DP + l8 * 4) * 4, qa = ka + TB * DP * 4;
      if (MODE == kScanDelta) {
        const uint32_t ga = ka + 2 * TB * DP * 4;
        f32x2 K[NCH * 2], A[CPT], B[CPT];
#pragma unroll
        for (int i = 0; i < CPT; ++i) A[i] = B[i] = 0ull;
#pragma unroll
        for (int c = 0; c < NCH; ++c) {
          f32x2 q0, q1, g0, g1;
          lds2(ka + c * 128, K[2 * c], K[2 * c + 1]);
          lds2(qa + c * 128, q0, q1);
          lds2(ga + c * 128, g0, g1);
#pragma unroll
          for (int i = 0; i < CPT; ++i) {
            S[i][2 * c] = mul2(S[i][2 * c], g0);
            S[i][2 * c + 1] = mul2(S[i][2 * c + 1], g1);
            A[i] = fma2(S[i][2 * c], K[2 * c], A[i]);
            B[i] = fma2(S[i][2 * c], q0, B[i]);
            A[i] = fma2(S[i][2 * c + 1], K[2 * c + 1], A[i]);
            B[i] = fma2(S[i][2 * c + 1], q1, B[i]);
          }
        }
        const float beta = st[off_s + 2 * t], kq = st[off_s + 2 * t + 1];
        float ra[CPT], rb[CPT];
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
          const float2 x = unpack2(A[i]), y = unpack2(B[i]);
          ra[i] = x.x + x.y;
          rb[i] = y.x + y.y;
        }
#pragma unroll
        for (int o = 4; o > 0; o >>= 1)
#pragma unroll
          for (int i = 0; i < CPT; ++i) {
            ra[i] += __shfl_xor_sync(0xffffffffu, ra[i], o);
            rb[i] += __shfl_xor_sync(0xffffffffu, rb[i], o);
          }
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
          const float u = beta * (st[off_v + t * cols + cg * CPT + i] - ra[i]);
          out[i] = fmaf(kq, u, rb[i]);
          const f32x2 u2 = pack2(u, u);
#pragma unroll
          for (int c = 0; c < NCH * 2; ++c) S[i][c] = fma2(K[c], u2, S[i][c]);
        }
      } else {
        const float fa = sh_gate[t], ib = sh_gate[TB + t], em = sh_gate[2 * TB + t];
        const f32x2 f2 = pack2(fa, fa), i2 = pack2(ib, ib);
        f32x2 B[CPT], vb[CPT], D = 0ull;
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
          const float v = st[off_v + t * cols + cg * CPT + i] * ib;
          vb[i] = pack2(v, v);
          B[i] = 0ull;
        }
#pragma unroll
        for (int c = 0; c < NCH; ++c) {
          f32x2 k0, k1, q0, q1;
          lds2(ka + c * 128, k0, k1);
          lds2(qa + c * 128, q0, q1);
#pragma unroll
          for (int i = 0; i < CPT; ++i) {
            S[i][2 * c] = fma2(k0, vb[i], mul2(S[i][2 * c], f2));
            S[i][2 * c + 1] = fma2(k1, vb[i], mul2(S[i][2 * c + 1], f2));
            B[i] = fma2(S[i][2 * c], q0, B[i]);
            B[i] = fma2(S[i][2 * c + 1], q1, B[i]);
          }
          N[2 * c] = fma2(k0, i2, mul2(N[2 * c], f2));
          N[2 * c + 1] = fma2(k1, i2, mul2(N[2 * c + 1], f2));
          D = fma2(N[2 * c], q0, D);
          D = fma2(N[2 * c + 1], q1, D);
        }
        const float2 dd = unpack2(D);
        const float den = fmaxf(fabsf(sum8(dd.x + dd.y)), em) + 1e-6f;
        const float inv = 1.0f / den;
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
          const float2 y = unpack2(B[i]);
          out[i] = sum8(y.x + y.y) * inv;
        }
      }
      if (!FUSED) {
        float* orow = a.out + (static_cast<int64_t>(t0 + t) * a.heads + head) * a.vdim + mycol;
#pragma unroll
        for (int i = 0; i < CPT; ++i)
          if (l8 == i && mycol + i < a.vdim) orow[i] = out[i];
      }
    }
    __syncthreads();       // the stage may be refilled
  }

#pragma unroll
  for (int i = 0; i < CPT; ++i)
    if (mycol + i < a.vdim) {
#pragma unroll
      for (int c = 0; c < NCH; ++c) {
        const float2 lo = unpack2(S[i][2 * c]), hi = unpack2(S[i][2 * c + 1]);
        *reinterpret_cast<float4*>(state + static_cast<int64_t>(mycol + i) * DP + c * 32 + l8 * 4) = make_float4(lo.x, lo.y, hi.x, hi.y);
      }
    }
  if (MODE == kScanMlstm) {
    // refresh the copies of the column blocks this CTA covers (the first column group of each)
    for (int b = col0 / kScanBlockCols; b < blocks && b * kScanBlockCols < col0 + cols; ++b) {
      if (cg != 0) break;
#pragma unroll
      for (int c = 0; c < NCH; ++c) {
        const float2 lo = unpack2(N[2 * c]), hi = unpack2(N[2 * c + 1]);
        *reinterpret_cast<float4*>(nstate + static_cast<int64_t>(b) * DP + c * 32 + l8 * 4) = make_float4(lo.x, lo.y, hi.x, hi.y);
      }
      if (threadIdx.x == 0) mstate[b] = run_max;
    }
  }
  if (FUSED) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < CPT; ++i)
      if (l8 == i && mycol + i < a.vdim) ss = out[i] * out[i];
    const float rstd = 1.0f / sqrtf(cta_sum(ss, red) / static_cast<float>(a.vdim) + a.eps);
    T* y = static_cast<T*>(a.y) + static_cast<int64_t>(t_begin) * a.ldy + static_cast<int64_t>(head) * a.vdim;
    const float* w = a.norm + static_cast<int64_t>(head) * a.norm_head_stride;
#pragma unroll
    for (int i = 0; i < CPT; ++i)
      if (l8 == i && mycol + i < a.vdim)
        y[mycol + i] = act_from_f<T>(out[i] * rstd * w[mycol + i] * sigmoid_f(rows_at<T>(a.gate, t_begin, head * a.vdim + mycol + i)));
  }
}

}  // namespace mdb

using namespace mdb;

namespace {

// at most 64 state registers per thread whatever the key size
constexpr int scan_cols_per_thread(int dim_pad) { return dim_pad <= 128 ? 4 : (dim_pad <= 256 ? 2 : 1); }
// column groups (of eight lanes) of a CTA that owns a whole head
constexpr int scan_fused_groups(int vdim, int cpt) { return ((vdim + cpt - 1) / cpt + 3) / 4 * 4; }

template <typename T, int MODE, int NCH, int CPT, int TB, bool FUSED>
int launch_scan_form(const mdb_scan_args& a, cudaStream_t st) {
  constexpr int DP = NCH * 32;
  int groups;                                     // column groups (of eight lanes) per CTA
  if (FUSED) groups = scan_fused_groups(a.vdim, CPT);
  else groups = kScanBlockCols / CPT;
  const int threads = groups * 8, cols = groups * CPT;
  if (FUSED && threads > kScanFusedThreads) return MDB_ERR_UNSUPPORTED;
  const int smem = 2 * scan_stage_floats(MODE, DP, TB, cols) * 4;
  if (smem > 200 * 1024) return MDB_ERR_UNSUPPORTED;
  static PerDeviceOnce attr_once;
  const int dev = attr_once.slot();
  if (dev < 0) return MDB_ERR_CUDA;
  if (!attr_once.done[dev]) {
    if (cudaFuncSetAttribute(scan_kernel<T, MODE, NCH, CPT, TB, FUSED>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) !=
        cudaSuccess)
      return MDB_ERR_CUDA;
    attr_once.done[dev] = true;
  }
  const dim3 grid(FUSED ? 1 : (a.vdim + cols - 1) / cols, a.heads, a.bs);
  return mdb_launch(scan_kernel<T, MODE, NCH, CPT, TB, FUSED>, grid, dim3(threads), smem, st, a, cols);
}

template <typename T, int MODE, int NCH>
int launch_scan_dim(const mdb_scan_args& a, cudaStream_t st) {
  constexpr int CPT = scan_cols_per_thread(NCH * 32);
  constexpr int TB = NCH <= 4 ? 16 : 8;
  if (a.fused) {
    if constexpr (NCH * 32 <= kScanFusedMaxDim) return launch_scan_form<T, MODE, NCH, CPT, 1, true>(a, st);
    else return MDB_ERR_UNSUPPORTED;
  }
  return launch_scan_form<float, MODE, NCH, CPT, TB, false>(a, st);     // the activation type plays no part here
}

template <typename T, int MODE>
int launch_scan(const mdb_scan_args& a, cudaStream_t st) {
  switch (a.dim_pad) {
    case 32: return launch_scan_dim<T, MODE, 1>(a, st);
    case 64: return launch_scan_dim<T, MODE, 2>(a, st);
    case 96: return launch_scan_dim<T, MODE, 3>(a, st);
    case 128: return launch_scan_dim<T, MODE, 4>(a, st);
    case 192: return launch_scan_dim<T, MODE, 6>(a, st);
    case 256: return launch_scan_dim<T, MODE, 8>(a, st);
    case 512: return launch_scan_dim<T, MODE, 16>(a, st);
    default: return MDB_ERR_UNSUPPORTED;
  }
}

bool seqs_ok(const int32_t* cu_q, const int32_t* start, const int32_t* slot) { return cu_q && start && slot; }

}  // namespace

extern "C" {

int mdb_scan_dim_pad(int dim) {
  static const int sizes[] = {32, 64, 96, 128, 192, 256, 512};
  for (int s : sizes)
    if (dim <= s) return s;
  return 0;
}

int mdb_scan_blocks(int vdim) { return (vdim + kScanBlockCols - 1) / kScanBlockCols; }

int mdb_scan_fusable(int dim_pad, int vdim) {
  return dim_pad <= kScanFusedMaxDim && scan_fused_groups(vdim, scan_cols_per_thread(dim_pad)) * 8 <= kScanFusedThreads ? 1 : 0;
}

int mdb_delta_prep(const mdb_delta_prep_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  mdb_delta_prep_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.bs >= 0 && a.heads > 0 && a.kv_heads > 0 && a.dim > 0 && a.vdim > 0 && a.taps > 0, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(a.heads % a.kv_heads == 0 && a.dim_pad >= a.dim, MDB_ERR_ARG);
  MDB_REQUIRE(a.channels == 2 * a.kv_heads * a.dim + a.heads * a.vdim, MDB_ERR_ARG);
  MDB_REQUIRE(rows_present(a.q) && rows_present(a.k) && rows_present(a.v) && rows_present(a.b), MDB_ERR_ARG);
  MDB_REQUIRE(a.conv_q && a.conv_k && a.conv_v && (a.conv_state || a.taps == 1) && a.row_seq &&
                  seqs_ok(a.cu_q, a.start, a.state_slot) && a.q_out && a.k_out && a.v_out && a.beta_out && a.kq_out,
              MDB_ERR_ARG);
  MDB_REQUIRE(a.copy_cols == 0 || (rows_present(a.copy) && a.copy_out && a.copy_cols % 4 == 0 && a.copy_ld % 4 == 0 && rows_ok(a.copy)),
              MDB_ERR_ARG);
  MDB_REQUIRE(a.taps <= kMaxTaps, MDB_ERR_UNSUPPORTED);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int units = a.kv_heads + a.heads + 1 + (a.copy_cols + 127) / 128;
  const dim3 grid(a.m, (units + kPrepWarps - 1) / kPrepWarps);
  int rc = a.dtype == MDB_F32 ? mdb_launch(delta_prep_kernel<float>, grid, dim3(kPrepWarps * 32), 0, st, a)
                              : mdb_launch(delta_prep_kernel<bf16>, grid, dim3(kPrepWarps * 32), 0, st, a);
  if (rc != MDB_OK || a.shift_state || a.taps < 2) return rc;
  const dim3 cgrid((a.channels + 255) / 256, a.bs);
  return a.dtype == MDB_F32 ? mdb_launch(conv_state_kernel<float>, cgrid, dim3(256), 0, st, a)
                            : mdb_launch(conv_state_kernel<bf16>, cgrid, dim3(256), 0, st, a);
}

int mdb_channel_decay(const float* x, int64_t ldx, const float* a_log, const float* dt_bias, float* g, int m, int heads,
                      int dim, int dim_pad, mdb_stream_t stream) {
  MDB_REQUIRE(m >= 0 && heads > 0 && dim > 0 && dim_pad >= dim, MDB_ERR_ARG);
  if (m == 0) return MDB_OK;
  MDB_REQUIRE(x && a_log && dt_bias && g && ldx >= static_cast<int64_t>(heads) * dim, MDB_ERR_ARG);
  const int64_t total = static_cast<int64_t>(m) * heads * dim_pad;
  const int64_t blocks = (total + 255) / 256;
  return mdb_launch(channel_decay_kernel, dim3(static_cast<int>(blocks < 148 * 16 ? blocks : 148 * 16)), dim3(256), 0,
                    static_cast<cudaStream_t>(stream), x, ldx, a_log, dt_bias, g, total, heads, dim, dim_pad);
}

int mdb_mlstm_prep(const mdb_mlstm_prep_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_mlstm_prep_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.heads > 0 && a.dim > 0 && a.dim_pad >= a.dim && a.vdim > 0 && a.cap > 0.f, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(rows_present(a.q) && rows_present(a.k) && rows_present(a.v) && rows_present(a.i) && rows_present(a.f) &&
                  a.bias_i && a.bias_f && a.q_out && a.k_out && a.v_out && a.log_i && a.log_f,
              MDB_ERR_ARG);
  const int items = a.heads * (a.dim_pad + a.vdim + 1);
  const dim3 grid(a.m, (items + 511) / 512);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return a.dtype == MDB_F32 ? mdb_launch(mlstm_prep_kernel<float>, grid, dim3(128), 0, st, a)
                            : mdb_launch(mlstm_prep_kernel<bf16>, grid, dim3(128), 0, st, a);
}

int mdb_scan(const mdb_scan_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_scan_args a = *args;
  MDB_REQUIRE(a.mode == MDB_SCAN_DELTA || a.mode == MDB_SCAN_MLSTM, MDB_ERR_ARG);
  MDB_REQUIRE(a.bs >= 0 && a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.vdim > 0, MDB_ERR_ARG);
  if (a.bs == 0) return MDB_OK;
  MDB_REQUIRE(a.q && a.k && a.v && a.s0 && a.s1 && a.state && seqs_ok(a.cu_q, a.start, a.state_slot), MDB_ERR_ARG);
  MDB_REQUIRE(a.mode != MDB_SCAN_MLSTM || (a.nstate && a.mstate && a.kv_heads == a.heads), MDB_ERR_ARG);
  if (a.fused) {
    MDB_REQUIRE(rows_present(a.gate) && a.norm && a.y, MDB_ERR_ARG);
    MDB_REQUIRE(a.mode != MDB_SCAN_DELTA || (rows_present(a.raw_decay) && a.a_log && a.dt_bias), MDB_ERR_ARG);
  } else {
    MDB_REQUIRE(a.out != nullptr && (a.mode != MDB_SCAN_DELTA || a.g != nullptr), MDB_ERR_ARG);
  }
  MDB_REQUIRE(mdb_aligned16(a.q) && mdb_aligned16(a.k) && mdb_aligned16(a.g) && mdb_aligned16(a.state) && mdb_aligned16(a.nstate) &&
                  a.state_slot_stride % 4 == 0,
              MDB_ERR_ALIGN);
  MDB_REQUIRE(a.heads <= 65535 && a.bs <= 65535, MDB_ERR_UNSUPPORTED);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a.dtype == MDB_F32)
    return a.mode == MDB_SCAN_DELTA ? launch_scan<float, kScanDelta>(a, st) : launch_scan<float, kScanMlstm>(a, st);
  return a.mode == MDB_SCAN_DELTA ? launch_scan<bf16, kScanDelta>(a, st) : launch_scan<bf16, kScanMlstm>(a, st);
}

}  // extern "C"
