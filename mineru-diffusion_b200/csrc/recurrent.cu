// Recurrent mixers with a matrix state per head: the gated delta rule with one decay per key channel, the mLSTM matrix
// memory, and plain linear recurrences with one decay per head, fixed or per token (lightning attention, Mamba-2).  A scan kernel each for prompts and their portions, one for single tokens; the state lives in fp32 in a slot
// per sequence and every product of the recurrence is an fp32 FMA (packed two at a time, fma.rn.f32x2).
//
// State layout: [slot][head][value column][key channel padded to a multiple of 64], so a value column is contiguous.
// The columns of a head are independent of one another (the delta rule's correction of a column only needs that
// column), so a CTA owns a block of columns: eight lanes (mLSTM prompts: sixteen) share a column, each holding every
// eighth (sixteenth) float4 of it in registers, CPT columns per thread.  k, q and the decays of a block of tokens come
// through a double-buffered shared-memory stage (cp.async).
//
// The read-out of the delta rule is rewritten so that both products with the old state share one reduction,
//   a = (g S)^T k,  b = (g S)^T q,  u = beta (v - a),  o = b + (k . q) u,  S <- g S + k u^T,
// and prompts take two tokens per reduction: with S' = g2 g1 S the second token's products are
//   a2 = S'^T k2 + ((g2 k1) . k2) u1,  b2 = S'^T q2 + ((g2 k1) . q2) u1,  S <- S' + (g2 k1) u1^T + k2 u2^T,
// the same number of FMAs per token with half the dependent shuffle reductions; these products of keys and queries are
// computed beforehand, with the decays.
//
// The linear recurrence S <- a S + b k v^T, o = S^T q + skip v is the mLSTM's scan with its gates given and no normaliser.
//
// mLSTM: the normaliser n is one more column of the state (its value is 1 for every token); the division by
// max(|n . q|, exp(-m)) + 1e-6 happens where the read-out is normalised.
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
__device__ __forceinline__ void lds2(const float* p, f32x2& a, f32x2& b) {      // four floats of shared memory
  const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p);
  a = v.x;
  b = v.y;
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
// Before the delta scan: short convolution + silu of q, k and v, unit norm of q and k, sigmoid of beta.
// Units of a row, one warp each: q and k of a head (together or apart), v of a head, one for beta, and, where the
// projection came as split-k slices, the copy of its low-rank columns for the GEMM that follows.
// ---------------------------------------------------------------------------
constexpr int kPrepWarps = 4;
constexpr int kMaxTaps = 16;

template <typename T, typename Args>
struct ConvCtx {
  const Args* a;
  int64_t row;
  int tloc, slot;      // token index inside this step's portion; state slot (-1: starts from zeros)
  int state_slot;      // the sequence's slot, whether or not its state counts
  // input of channel `col` of projection `src`, `back` tokens ago
  __device__ __forceinline__ float at(const mdb_rows& src, int col, int channel, int back) const {
    if (back <= tloc) return rows_at<T>(src, row - back, col);
    const int idx = a->taps - 1 - (back - tloc);
    if (slot < 0 || idx < 0) return 0.f;
    return act_to_f(static_cast<const T*>(a->conv_state)[slot * a->conv_slot_stride + static_cast<int64_t>(idx) * a->channels + channel]);
  }
  __device__ __forceinline__ float conv_silu(const mdb_rows& src, const float* w, int col, int channel, float bias = 0.f) const {
    float acc = bias;
    for (int j = 0; j < a->taps; ++j) acc = fmaf(w[static_cast<int64_t>(col) * a->taps + j], at(src, col, channel, a->taps - 1 - j), acc);
    return acc / (1.0f + expf(-acc));
  }
  // one-token portions move the convolution state along: the caller owns the channel
  __device__ __forceinline__ void shift(const mdb_rows& src, int col, int channel) const {
    if (!a->shift_state || a->taps < 2) return;
    T* st = static_cast<T*>(a->conv_state) + state_slot * a->conv_slot_stride + channel;
    float keep[kMaxTaps];
#pragma unroll 1
    for (int j = 0; j < a->taps - 1; ++j) keep[j] = at(src, col, channel, a->taps - 2 - j);
#pragma unroll 1
    for (int j = 0; j < a->taps - 1; ++j) st[static_cast<int64_t>(j) * a->channels] = act_from_f<T>(keep[j]);
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
  const ConvCtx<T, mdb_delta_prep_args> cx = {&a, row, static_cast<int>(row) - a.cu_q[seq], a.start[seq] == 0 ? -1 : slot, slot};
  if (unit < a.kv_heads) {
    float* qo = a.q_out + (row * a.kv_heads + unit) * a.dim_pad;
    float* ko = a.k_out + (row * a.kv_heads + unit) * a.dim_pad;
    const int kq_channels = a.kv_heads * a.dim;
    float sq = 0.f, sk = 0.f;
    for (int d = lane; d < a.dim_pad; d += 32) {
      float q = 0.f, k = 0.f;
      if (d < a.dim) {
        const int col = unit * a.dim + d;
        q = cx.conv_silu(a.q, a.conv_q, col, col);
        k = cx.conv_silu(a.k, a.conv_k, col, kq_channels + col);
        cx.shift(a.q, col, col);
        cx.shift(a.k, col, kq_channels + col);
      }
      qo[d] = q;
      ko[d] = k;
      sq += q * q;
      sk += k * k;
    }
    const float rq = (1.0f / sqrtf(warp_sum(sq) + 1e-6f)) * (1.0f / sqrtf(static_cast<float>(a.dim)));
    const float rk = 1.0f / sqrtf(warp_sum(sk) + 1e-6f);
    for (int d = lane; d < a.dim_pad; d += 32) {       // a lane re-reads what it wrote itself
      qo[d] *= rq;
      ko[d] *= rk;
    }
    return;
  }
  const int vu = unit - a.kv_heads;
  if (vu < a.heads) {
    float* vo = a.v_out + (row * a.heads + vu) * a.vdim;
    for (int d = lane; d < a.vdim; d += 32) {
      const int col = vu * a.vdim + d, channel = 2 * a.kv_heads * a.dim + col;
      const float v = cx.conv_silu(a.v, a.conv_v, col, channel);
      cx.shift(a.v, col, channel);
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

// silu; the approximate division and exponential are good to a few units in the last place of fp32, and a large negative
// argument (whose exponential leaves the range of the fast division) gives 0
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-fmaxf(z, -80.f))); }
__device__ __forceinline__ float4 silu4(float4 z) { return make_float4(silu_fast(z.x), silu_fast(z.y), silu_fast(z.z), silu_fast(z.w)); }

// The same work for heads of at most 128 channels and up to four taps, sizes in multiples of four: a lane owns four
// channels and walks `run` consecutive rows with the last inputs in registers, so every input is read once.
template <typename T, bool PARTS>
struct ConvWindow {
  float4 x[3];         // inputs 3, 2 and 1 tokens ago
  float4 w[4];         // taps of the four channels: w[j] belongs to the input 3 - j tokens ago
  __device__ __forceinline__ void load_taps(const float* weights, int col, int taps) {
    if (taps == 4) {
      const float4* p = reinterpret_cast<const float4*>(weights + static_cast<int64_t>(col) * 4);
      const float4 a = p[0], b = p[1], c = p[2], d = p[3];
      w[0] = make_float4(a.x, b.x, c.x, d.x); w[1] = make_float4(a.y, b.y, c.y, d.y);
      w[2] = make_float4(a.z, b.z, c.z, d.z); w[3] = make_float4(a.w, b.w, c.w, d.w);
      return;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = j - (4 - taps);
      float e[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) e[c] = t >= 0 ? weights[static_cast<int64_t>(col + c) * taps + t] : 0.f;
      w[j] = make_float4(e[0], e[1], e[2], e[3]);
    }
  }
  template <typename Args>
  __device__ __forceinline__ void refill(const Args& a, const mdb_rows& src, int64_t row, int tloc, int slot, int col, int channel) {
#pragma unroll
    for (int back = 1; back <= 3; ++back) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (back < a.taps) {
        if (back <= tloc) v = rows_at4_of<T, PARTS>(src, row - back, col);
        else if (slot >= 0)
          v = act_load4(static_cast<const T*>(a.conv_state) + slot * a.conv_slot_stride +
                        static_cast<int64_t>(a.taps - 1 - (back - tloc)) * a.channels + channel);
      }
      x[3 - back] = v;
    }
  }
  __device__ __forceinline__ float4 step(float4 now, float4 bias = make_float4(0.f, 0.f, 0.f, 0.f)) {
    float4 y;
    y.x = fmaf(w[3].x, now.x, fmaf(w[2].x, x[2].x, fmaf(w[1].x, x[1].x, fmaf(w[0].x, x[0].x, bias.x))));
    y.y = fmaf(w[3].y, now.y, fmaf(w[2].y, x[2].y, fmaf(w[1].y, x[1].y, fmaf(w[0].y, x[0].y, bias.y))));
    y.z = fmaf(w[3].z, now.z, fmaf(w[2].z, x[2].z, fmaf(w[1].z, x[1].z, fmaf(w[0].z, x[0].z, bias.z))));
    y.w = fmaf(w[3].w, now.w, fmaf(w[2].w, x[2].w, fmaf(w[1].w, x[1].w, fmaf(w[0].w, x[0].w, bias.w))));
    x[0] = x[1]; x[1] = x[2]; x[2] = now;
    return silu4(y);
  }
  // one-token portions: the last taps - 1 inputs back into the slot
  template <typename Args>
  __device__ __forceinline__ void save(const Args& a, int slot, int channel) const {
    T* st = static_cast<T*>(a.conv_state) + slot * a.conv_slot_stride + channel;
    for (int j = 0; j < a.taps - 1; ++j) {
      const int i = 3 - (a.taps - 1) + j;          // oldest first
      act_store4(st + static_cast<int64_t>(j) * a.channels, i == 0 ? x[0] : (i == 1 ? x[1] : x[2]));
    }
  }
};
__device__ __forceinline__ float dot4(float4 a, float4 b) { return a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w; }
__device__ __forceinline__ float4 scale4(float4 a, float s) { return make_float4(a.x * s, a.y * s, a.z * s, a.w * s); }

template <typename T, bool PARTS>
__global__ void __launch_bounds__(kPrepWarps * 32, 7) delta_prep_rows_kernel(const mdb_delta_prep_args a, const int run) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, c = lane * 4;
  const int unit = blockIdx.x * kPrepWarps + (threadIdx.x >> 5);
  const int64_t row0 = static_cast<int64_t>(blockIdx.y) * run, row1 = min(row0 + run, static_cast<int64_t>(a.m));
  const int vblocks = (a.vdim + 127) / 128;        // a head's values in blocks of 128
  const int qk_units = 2 * a.kv_heads, kc = a.kv_heads * a.dim;
  if (unit < qk_units + a.heads * vblocks) {
    const int stream = unit < a.kv_heads ? 0 : (unit < qk_units ? 1 : 2);      // q, k or v
    const int vu = unit - qk_units, head = stream == 2 ? vu / vblocks : unit - stream * a.kv_heads;
    const int hc = stream == 2 ? (vu % vblocks) * 128 + c : c;       // first of the lane's channels in its head
    const int dim = stream == 2 ? a.vdim : a.dim;
    const bool live = hc < dim;
    const int col = head * dim + hc, channel = stream * kc + col;
    // by value: a reference picked at run time would be read through memory at every use
    mdb_rows src = a.q;
    if (stream == 1) src = a.k;
    if (stream == 2) src = a.v;
    ConvWindow<T, PARTS> win;
    if (live) win.load_taps(stream == 0 ? a.conv_q : (stream == 1 ? a.conv_k : a.conv_v), col, a.taps);
    const float unit_scale = stream == 0 ? 1.0f / sqrtf(static_cast<float>(a.dim)) : 1.0f;
    const int out_dim = stream == 2 ? a.vdim : a.dim_pad, out_heads = stream == 2 ? a.heads : a.kv_heads;
    float* out = (stream == 0 ? a.q_out : (stream == 1 ? a.k_out : a.v_out)) + static_cast<int64_t>(head) * out_dim + hc;
    const int64_t out_ld = static_cast<int64_t>(out_heads) * out_dim;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    int seq = -1, slot = -1;
    for (int64_t row = row0; row < row1; ++row) {
      const int s = a.row_seq[row];
      const float4 in = live ? rows_at4_of<T, PARTS>(src, row, col) : zero;
      if (s != seq) {
        seq = s;
        slot = a.state_slot[s];
        if (slot >= a.num_slots) {
          if (lane == 0) report_status(MDB_STATUS_BAD_SLOT);
          slot = -1;
        }
        if (slot >= 0 && live)
          win.refill(a, src, row, static_cast<int>(row) - a.cu_q[s], a.start[s] == 0 ? -1 : slot, col, channel);
      }
      if (slot < 0) continue;
      float4 y = zero;
      if (live) {
        y = win.step(in);
        if (a.shift_state && a.taps > 1) win.save(a, slot, channel);
      }
      if (stream < 2) y = scale4(y, (1.0f / sqrtf(warp_sum(dot4(y, y)) + 1e-6f)) * unit_scale);
      if (hc < out_dim) *reinterpret_cast<float4*>(out + row * out_ld) = y;
    }
    return;
  }
  const int rest = unit - qk_units - a.heads * vblocks;
  if (rest == 0) {
    const int n = static_cast<int>(row1 - row0) * a.heads;
#pragma unroll 4
    for (int i = lane; i < n; i += 32) {
      const int64_t row = row0 + i / a.heads;
      a.beta_out[row * a.heads + i % a.heads] = sigmoid_f(rows_at<T>(a.b, row, i % a.heads));
    }
    return;
  }
  const int cc = (rest - 1) * 128 + c;
  if (cc < a.copy_cols)
    for (int64_t row = row0; row < row1; ++row)
      act_store4(static_cast<T*>(a.copy_out) + row * a.copy_ld + cc, rows_at4_of<T, PARTS>(a.copy, row, cc));
}

// Where a convolution channel's input comes from: the projection, and `channel` turned into a column of it.
__device__ __forceinline__ const mdb_rows& conv_source(const mdb_delta_prep_args& a, int& channel) {
  const int kc = a.kv_heads * a.dim;
  if (channel < kc) return a.q;
  channel -= kc;
  if (channel < kc) return a.k;
  channel -= kc;
  return a.v;
}
__device__ __forceinline__ const mdb_rows& conv_source(const mdb_decay_prep_args& a, int& channel) {
  const int kc = a.kv_heads * a.dim, vc = a.heads * a.vdim;
  if (channel < vc) return a.v;
  channel -= vc;
  if (channel < kc) return a.k;
  channel -= kc;
  return a.q;
}

// The last taps - 1 inputs of every channel after a step of arbitrary portions: one thread per (sequence, channel).
template <typename T, typename Args>
__global__ void __launch_bounds__(256) conv_state_kernel(const Args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.y;
  const int channel = blockIdx.x * 256 + threadIdx.x;
  const int slot = a.state_slot[seq];
  if (slot < 0 || slot >= a.num_slots || channel >= a.channels) return;
  const int t0 = a.cu_q[seq], n = a.cu_q[seq + 1] - t0;
  if (n <= 0) return;
  int col = channel;
  const mdb_rows& src = conv_source(a, col);
  const ConvCtx<T, Args> cx = {&a, t0 + n - 1, n - 1, a.start[seq] == 0 ? -1 : slot, slot};
  float keep[kMaxTaps];
#pragma unroll 1
  for (int j = 0; j < a.taps - 1; ++j) keep[j] = cx.at(src, col, channel, a.taps - 2 - j);
  T* st = static_cast<T*>(a.conv_state) + slot * a.conv_slot_stride + channel;
#pragma unroll 1
  for (int j = 0; j < a.taps - 1; ++j) st[static_cast<int64_t>(j) * a.channels] = act_from_f<T>(keep[j]);
}

// A warp per (row, head).  g = exp(-exp(A_log) * softplus(x + dt_bias)), laid out [row][head][dim_pad] (padding
// channels: 1), and the scalars of the scan, [row][head][4] = (k . q, (g k_prev) . k, (g k_prev) . q, beta): the middle two
// are the products with the token before and exist for the odd tokens of a portion.  VEC: head rows of x start on 16-byte boundaries.
template <bool VEC>
__global__ void __launch_bounds__(128) channel_decay_kernel(const mdb_decay_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int64_t row = blockIdx.x;
  const bool odd = ((static_cast<int>(row) - a.cu_q[a.row_seq[row]]) & 1) != 0;
#pragma unroll 2
  for (int head = blockIdx.y * 4 + (threadIdx.x >> 5); head < a.heads; head += gridDim.y * 4) {
    const float* x = a.x + row * a.ldx + static_cast<int64_t>(head) * a.dim;
    const float* bias = a.dt_bias + static_cast<int64_t>(head) * a.dim;
    float* g = a.g + (row * a.heads + head) * a.dim_pad;
    const int kvh = head / (a.heads / a.kv_heads);
    const float* k = a.k + (row * a.kv_heads + kvh) * a.dim_pad;
    const float* q = a.q + (row * a.kv_heads + kvh) * a.dim_pad;
    const float* kp = k - static_cast<int64_t>(a.kv_heads) * a.dim_pad;      // read for odd tokens only
    const float rate = -expf(a.a_log[head]);
    float kq = 0.f, ck = 0.f, cq = 0.f;
    for (int c = lane * 4; c < a.dim_pad; c += 128) {
      float xv[4], bv[4], r[4];
      if (VEC && c + 4 <= a.dim) {
        const float4 x4 = *reinterpret_cast<const float4*>(x + c), b4 = *reinterpret_cast<const float4*>(bias + c);
        xv[0] = x4.x; xv[1] = x4.y; xv[2] = x4.z; xv[3] = x4.w;
        bv[0] = b4.x; bv[1] = b4.y; bv[2] = b4.z; bv[3] = b4.w;
      } else {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          xv[i] = c + i < a.dim ? x[c + i] : 0.f;
          bv[i] = c + i < a.dim ? bias[c + i] : 0.f;
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) r[i] = c + i < a.dim ? expf(rate * softplus_f(xv[i] + bv[i])) : 1.f;
      *reinterpret_cast<float4*>(g + c) = make_float4(r[0], r[1], r[2], r[3]);
      const float4 k1 = *reinterpret_cast<const float4*>(k + c), q1 = *reinterpret_cast<const float4*>(q + c);
      kq += dot4(k1, q1);
      if (odd) {
        const float4 k0 = *reinterpret_cast<const float4*>(kp + c);
        const float4 e = make_float4(r[0] * k0.x, r[1] * k0.y, r[2] * k0.z, r[3] * k0.w);
        ck += dot4(e, k1);
        cq += dot4(e, q1);
      }
    }
    kq = warp_sum(kq);
    if (odd) {
      ck = warp_sum(ck);
      cq = warp_sum(cq);
    }
    if (lane == 0)
      *reinterpret_cast<float4*>(a.scalars + 4 * (row * a.heads + head)) = make_float4(kq, ck, cq, a.beta[row * a.heads + head]);
  }
}

// Before the mLSTM scan: q scaled, k, v as fp32 rows (key channels padded with zeros), and the two log gates.  Work
// items of four channels; VEC: head rows of the projections start on 16-byte boundaries.
template <typename T, bool VEC, bool PARTS>
__global__ void __launch_bounds__(256) mlstm_prep_kernel(const mdb_mlstm_prep_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int nq = a.heads * a.dim_pad, nv = a.heads * a.vdim;
  const int iq = nq / 4, iv = (nv + 3) / 4;
  const float scale = 1.0f / sqrtf(static_cast<float>(a.dim));
  for (int i = blockIdx.y * 256 + threadIdx.x; i < iq + iv + a.heads; i += gridDim.y * 256) {
    if (i < iq) {
      const int h = i * 4 / a.dim_pad, d = i * 4 % a.dim_pad;
      float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q;
      if (VEC) {
        if (d < a.dim) {
          q = rows_at4_of<T, PARTS>(a.q, row, h * a.dim + d);
          k = rows_at4_of<T, PARTS>(a.k, row, h * a.dim + d);
        }
      } else {
        float* qe = &q.x;
        float* ke = &k.x;
        for (int e = 0; e < 4 && d + e < a.dim; ++e) {
          qe[e] = rows_at<T>(a.q, row, h * a.dim + d + e);
          ke[e] = rows_at<T>(a.k, row, h * a.dim + d + e);
        }
      }
      *reinterpret_cast<float4*>(a.q_out + row * nq + i * 4) = make_float4(q.x * scale, q.y * scale, q.z * scale, q.w * scale);
      *reinterpret_cast<float4*>(a.k_out + row * nq + i * 4) = k;
    } else if (i < iq + iv) {
      const int c = (i - iq) * 4;
      if (VEC) {
        *reinterpret_cast<float4*>(a.v_out + row * nv + c) = rows_at4_of<T, PARTS>(a.v, row, c);
      } else {
        for (int e = c; e < c + 4 && e < nv; ++e) a.v_out[row * nv + e] = rows_at<T>(a.v, row, e);
      }
    } else {
      const int h = i - iq - iv;
      const float zi = rows_at<T>(a.i, row, h) + a.bias_i[h], zf = rows_at<T>(a.f, row, h) + a.bias_f[h];
      a.log_i[row * a.heads + h] = a.cap * tanhf(zi / a.cap);
      a.log_f[row * a.heads + h] = -softplus_f(-(a.cap * tanhf(zf / a.cap)));
    }
  }
}

// ---------------------------------------------------------------------------
// Before the decay scan: silu or short convolution + silu of v, k and q, and the two scalars of a head.  Work items of a row:
// channels of v, of k, of q (padding channels: zeros), then one per head for the scalars.
// ---------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ void decay_prep_scalars(const mdb_decay_prep_args& a, int64_t row, int head) {
  constexpr float kMinLog = -104.0f;         // e^-104 is 0 in fp32; the bound keeps the sums of logs of a chunk small
  float decay, step = 1.0f;
  if (rows_present(a.dt)) {
    step = softplus_f(rows_at<T>(a.dt, row, head) + a.dt_bias[head]);
    const float log_decay = -expf(a.a_log[head]) * step;
    decay = a.for_chunks ? fmaxf(log_decay, kMinLog) : expf(log_decay);
  } else {
    decay = a.for_chunks ? fmaxf(logf(a.decay_const[head]), kMinLog) : a.decay_const[head];
  }
  a.decay_out[row * a.heads + head] = decay;
  a.step_out[row * a.heads + head] = step;
}

template <typename T, typename O>
__global__ void __launch_bounds__(256) decay_prep_kernel(const mdb_decay_prep_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int seq = a.row_seq[row];
  const int slot = a.state_slot[seq];
  if (slot < 0) return;
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0) report_status(MDB_STATUS_BAD_SLOT);
    return;
  }
  int i = blockIdx.y * 256 + threadIdx.x;
  const int nv = a.heads * a.vdim, nk = a.kv_heads * a.dim_pad, kc = a.kv_heads * a.dim;
  if (i >= nv + 2 * nk) {
    if (i - nv - 2 * nk < a.heads) decay_prep_scalars<T>(a, row, i - nv - 2 * nk);
    return;
  }
  const int stream = i < nv ? 0 : (i < nv + nk ? 1 : 2);
  i -= stream == 0 ? 0 : (stream == 1 ? nv : nv + nk);
  const mdb_rows& src = stream == 0 ? a.v : (stream == 1 ? a.k : a.q);
  O* out = static_cast<O*>(stream == 0 ? a.v_out : (stream == 1 ? a.k_out : a.q_out)) + row * (stream == 0 ? nv : nk) + i;
  int col = i;
  if (stream > 0) {
    const int d = i % a.dim_pad;
    if (d >= a.dim) {
      *out = act_from_f<O>(0.f);
      return;
    }
    col = i / a.dim_pad * a.dim + d;
  }
  if (a.taps == 0) {
    const float x = rows_at<T>(src, row, col);
    *out = act_from_f<O>(x / (1.0f + expf(-x)));
    return;
  }
  const ConvCtx<T, mdb_decay_prep_args> cx = {&a, row, static_cast<int>(row) - a.cu_q[seq], a.start[seq] == 0 ? -1 : slot, slot};
  const int channel = col + (stream == 0 ? 0 : (stream == 1 ? nv : nv + kc));
  const float* w = a.conv + static_cast<int64_t>(channel - col) * a.taps;
  *out = act_from_f<O>(cx.conv_silu(src, w, col, channel, a.conv_bias[channel]));
  cx.shift(src, col, channel);
}

// Four activations as they lie in memory.
template <typename T> struct ActRaw;
template <> struct ActRaw<float> { typedef float4 type; };
template <> struct ActRaw<bf16> { typedef uint2 type; };
__device__ __forceinline__ float4 act_raw4(float4 v) { return v; }
__device__ __forceinline__ float4 act_raw4(uint2 u) {
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}

// Sizes in multiples of four and up to four taps: a thread owns four channels and walks `run` consecutive rows with the last
// inputs in registers.
constexpr int kDecayPrepThreads = 128;
template <typename T, typename O, bool PARTS>
__global__ void __launch_bounds__(kDecayPrepThreads, 8) decay_prep_rows_kernel(const mdb_decay_prep_args a, const int run) {
  pdl_launch_dependents();
  pdl_wait();
  int i = blockIdx.x * kDecayPrepThreads + threadIdx.x;
  const int64_t row0 = static_cast<int64_t>(blockIdx.y) * run, row1 = min(row0 + run, static_cast<int64_t>(a.m));
  const int nv = a.heads * a.vdim, nk = a.kv_heads * a.dim_pad, kc = a.kv_heads * a.dim;
  const int iv = nv / 4, ik = nk / 4;
  if (i >= iv + 2 * ik) {
    i -= iv + 2 * ik;
    if (i < a.heads)
      for (int64_t row = row0; row < row1; ++row) decay_prep_scalars<T>(a, row, i);
    return;
  }
  const int stream = i < iv ? 0 : (i < iv + ik ? 1 : 2);
  i -= stream == 0 ? 0 : (stream == 1 ? iv : iv + ik);
  mdb_rows src = a.v;
  if (stream == 1) src = a.k;
  if (stream == 2) src = a.q;
  const int64_t out_ld = stream == 0 ? nv : nk;
  O* out = static_cast<O*>(stream == 0 ? a.v_out : (stream == 1 ? a.k_out : a.q_out)) + i * 4;
  int col = i * 4;
  if (stream > 0) {
    const int d = i * 4 % a.dim_pad;
    if (d >= a.dim) {
      for (int64_t row = row0; row < row1; ++row) act_store4(out + row * out_ld, make_float4(0.f, 0.f, 0.f, 0.f));
      return;
    }
    col = i * 4 / a.dim_pad * a.dim + d;
  }
  if (a.taps == 0) {
#pragma unroll 4
    for (int64_t row = row0; row < row1; ++row) act_store4(out + row * out_ld, silu4(rows_at4_of<T, PARTS>(src, row, col)));
    return;
  }
  const int channel = col + (stream == 0 ? 0 : (stream == 1 ? nv : nv + kc));
  ConvWindow<T, PARTS> win;
  win.load_taps(a.conv, channel, a.taps);
  const float4 bias = *reinterpret_cast<const float4*>(a.conv_bias + channel);
  int seq = -1, slot = -1;
  constexpr int kAhead = PARTS ? 1 : 4;        // rows whose inputs are requested together
  typedef typename ActRaw<T>::type Raw;
  for (int64_t row = row0; row < row1;) {
    if (!PARTS && row + kAhead <= row1 && a.row_seq[row] == seq && a.row_seq[row + kAhead - 1] == seq && slot >= 0 && !a.shift_state) {
      Raw in[kAhead];
      const T* x = static_cast<const T*>(src.x) + row * src.ld + src.col + col;
#pragma unroll
      for (int r = 0; r < kAhead; ++r) in[r] = *reinterpret_cast<const Raw*>(x + r * src.ld);
#pragma unroll
      for (int r = 0; r < kAhead; ++r) act_store4(out + (row + r) * out_ld, win.step(act_raw4(in[r]), bias));
      row += kAhead;
      continue;
    }
    const int s = a.row_seq[row];
    if (s != seq) {
      seq = s;
      slot = a.state_slot[s];
      if (slot >= a.num_slots) {
        report_status(MDB_STATUS_BAD_SLOT);
        slot = -1;
      }
      if (slot >= 0) win.refill(a, src, row, static_cast<int>(row) - a.cu_q[s], a.start[s] == 0 ? -1 : slot, col, channel);
    }
    if (slot >= 0) {
      act_store4(out + row * out_ld, win.step(rows_at4_of<T, PARTS>(src, row, col), bias));
      if (a.shift_state && a.taps > 1) win.save(a, slot, channel);
    }
    ++row;
  }
}

// ---------------------------------------------------------------------------
// The scan
// ---------------------------------------------------------------------------
enum { kScanDelta = MDB_SCAN_DELTA, kScanMlstm = MDB_SCAN_MLSTM, kScanDecay = MDB_SCAN_DECAY };
constexpr int kScanFusedThreads = 512, kScanFusedMaxDim = 256;
constexpr int kScanBlockCols = 16;       // granularity of the copies of the mLSTM maximum; narrowest block of a prompt CTA
constexpr int kScanTokens = 16;          // tokens of a stage of the prompt form (even)

// floats of one stage: k, q (and the decays) of tb tokens, their values for `cols` columns, four scalars per token
__host__ __device__ constexpr int scan_stage_floats(int mode, int dp, int tb, int cols) {
  return tb * ((mode == kScanDelta ? 3 : 2) * dp + cols + 4);
}

template <int NCH, int CPT>
struct ScanState {
  f32x2 v[CPT][NCH * 2];
  // column col0 + i of a head's state (columns from `columns` on: zeros)
  __device__ __forceinline__ void load(const float* state, int col0, int columns, int l8, bool fresh) {
#pragma unroll
    for (int i = 0; i < CPT; ++i)
#pragma unroll
      for (int c = 0; c < NCH; ++c) {
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && col0 + i < columns)
          x = *reinterpret_cast<const float4*>(state + static_cast<int64_t>(col0 + i) * (NCH * 32) + c * 32 + l8 * 4);
        v[i][2 * c] = pack2(x.x, x.y);
        v[i][2 * c + 1] = pack2(x.z, x.w);
      }
  }
  __device__ __forceinline__ void store(float* state, int col0, int columns, int l8) const {
#pragma unroll
    for (int i = 0; i < CPT; ++i)
      if (col0 + i < columns) {
#pragma unroll
        for (int c = 0; c < NCH; ++c) {
          const float2 lo = unpack2(v[i][2 * c]), hi = unpack2(v[i][2 * c + 1]);
          *reinterpret_cast<float4*>(state + static_cast<int64_t>(col0 + i) * (NCH * 32) + c * 32 + l8 * 4) =
              make_float4(lo.x, lo.y, hi.x, hi.y);
        }
      }
  }
};

// What a CTA of the prompt form works on: COLS columns of one head of one sequence.
struct ScanJob {
  bool live, fresh;
  int head, kvh, slot, t_begin, t_end, col0, columns;
  float* state;       // the head's columns
};
template <int MODE, int DP, int COLS>
__device__ __forceinline__ ScanJob scan_job(const mdb_scan_args& a) {
  ScanJob w = {};
  const int seq = blockIdx.z;
  w.head = blockIdx.y;
  w.col0 = blockIdx.x * COLS;
  w.slot = a.state_slot[seq];
  if (w.slot < 0) return w;
  if (w.slot >= a.num_slots) {
    if (threadIdx.x == 0) report_status(MDB_STATUS_BAD_SLOT);
    return w;
  }
  w.t_begin = a.cu_q[seq];
  w.t_end = a.cu_q[seq + 1];
  w.live = w.t_end > w.t_begin;
  w.fresh = a.start[seq] == 0;
  w.kvh = w.head / (a.heads / a.kv_heads);
  w.columns = a.vdim + (MODE == kScanMlstm ? 1 : 0);
  w.state = a.state + w.slot * a.state_slot_stride + static_cast<int64_t>(w.head) * w.columns * DP;
  return w;
}

template <int MODE, int DP, int COLS>
struct ScanStage {
  static constexpr int TB = kScanTokens, VEC = MODE == kScanDelta ? 3 : 2;
  static constexpr int OFF_V = TB * VEC * DP, OFF_S = OFF_V + TB * COLS, FLOATS = scan_stage_floats(MODE, DP, TB, COLS);
  // requests the operands of tokens [t0, t0 + TB) into the buffer at st
  static __device__ __forceinline__ void fill(const mdb_scan_args& a, const ScanJob& w, int t0, float* st) {
    const int n = min(TB, w.t_end - t0), step = blockDim.x;
    const uint32_t base = smem_u32(st);
    for (int i = threadIdx.x; i < n * (DP / 4); i += step) {
      const int t = i / (DP / 4), c = i % (DP / 4);
      const int64_t krow = (static_cast<int64_t>(t0 + t) * a.kv_heads + w.kvh) * DP + c * 4;
      cp_async16(base + (t * DP + c * 4) * 4, a.k + krow);
      cp_async16(base + ((TB + t) * DP + c * 4) * 4, a.q + krow);
      if (MODE == kScanDelta)
        cp_async16(base + ((2 * TB + t) * DP + c * 4) * 4, a.g + (static_cast<int64_t>(t0 + t) * a.heads + w.head) * DP + c * 4);
    }
    for (int i = threadIdx.x; i < n * COLS; i += step) {
      const int t = i / COLS, c = i % COLS;
      if (w.col0 + c < a.vdim)
        cp_async4(base + (OFF_V + t * COLS + c) * 4, a.v + (static_cast<int64_t>(t0 + t) * a.heads + w.head) * a.vdim + w.col0 + c);
      else
        st[OFF_V + t * COLS + c] = MODE == kScanMlstm && w.col0 + c == a.vdim ? 1.f : 0.f;
    }
    for (int i = threadIdx.x; i < n; i += step) {
      const int64_t th = static_cast<int64_t>(t0 + i) * a.heads + w.head;
      const uint32_t dst = base + (OFF_S + 4 * i) * 4;
      if (MODE == kScanDelta) {
        cp_async16(dst, a.scalars + 4 * th);
      } else {
        cp_async4(dst, a.s0 + th);
        cp_async4(dst + 4, a.s1 + th);
      }
    }
    if (n & 1) {
      // the missing second token of the last pair changes nothing: no key, no query, no decay
      for (int i = threadIdx.x; i < DP; i += step) {
        st[n * DP + i] = st[(TB + n) * DP + i] = 0.f;
        if (MODE == kScanDelta) st[(2 * TB + n) * DP + i] = 1.f;
      }
      for (int i = threadIdx.x; i < COLS; i += step) st[OFF_V + n * COLS + i] = 0.f;
      if (threadIdx.x < 4) st[OFF_S + 4 * n + threadIdx.x] = MODE == kScanDecay && threadIdx.x == 0 ? 1.f : 0.f;
    }
    cp_async_commit();
  }
  // on return the tokens from t0 on are in buffer buf for the whole CTA, and the next ones have been requested
  static __device__ __forceinline__ void turn(const mdb_scan_args& a, const ScanJob& w, int t0, float* smem, int buf) {
    if (t0 + TB < w.t_end) {
      fill(a, w, t0 + TB, smem + (buf ^ 1) * FLOATS);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
  }
};

// Delta rule, prompt form: portions of any length, two tokens at a time, eight lanes per column.
template <int NCH, int CPT, int COLS>
__global__ void __launch_bounds__(COLS / CPT * 8) delta_scan_kernel(const mdb_scan_args a) {
  constexpr int DP = NCH * 32;
  using Stage = ScanStage<kScanDelta, DP, COLS>;
  constexpr int TB = Stage::TB;
  constexpr bool KEEP_K = NCH <= 8;      // the keys of a pair stay in registers between the two passes
  extern __shared__ __align__(16) float scan_smem[];
  pdl_launch_dependents();
  pdl_wait();
  const ScanJob w = scan_job<kScanDelta, DP, COLS>(a);
  if (!w.live) return;
  const int l8 = threadIdx.x & 7, cg = threadIdx.x >> 3, mycol = w.col0 + cg * CPT;
  ScanState<NCH, CPT> S;
  S.load(w.state, mycol, w.columns, l8, w.fresh);
  Stage::fill(a, w, w.t_begin, scan_smem);
  int buf = 0;
  for (int t0 = w.t_begin; t0 < w.t_end; t0 += TB, buf ^= 1) {
    const int n = min(TB, w.t_end - t0);
    Stage::turn(a, w, t0, scan_smem, buf);
    const float* st = scan_smem + buf * Stage::FLOATS;
    for (int t = 0; t < n; t += 2) {
      const float* ka = st + t * DP + l8 * 4;
      const float* qa = ka + TB * DP;
      const float* ga = ka + 2 * TB * DP;
      f32x2 K1[KEEP_K ? NCH * 2 : 1], K2[KEEP_K ? NCH * 2 : 1];
      f32x2 A1[CPT], B1[CPT], A2[CPT], B2[CPT];
#pragma unroll
      for (int i = 0; i < CPT; ++i) A1[i] = B1[i] = A2[i] = B2[i] = 0ull;
#pragma unroll
      for (int c = 0; c < NCH; ++c) {
        f32x2 k1[2], q1[2], g1[2], k2[2], q2[2], g2[2];
        lds2(ka + c * 32, k1[0], k1[1]);
        lds2(qa + c * 32, q1[0], q1[1]);
        lds2(ga + c * 32, g1[0], g1[1]);
        lds2(ka + DP + c * 32, k2[0], k2[1]);
        lds2(qa + DP + c * 32, q2[0], q2[1]);
        lds2(ga + DP + c * 32, g2[0], g2[1]);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (KEEP_K) {
            K1[KEEP_K ? 2 * c + e : 0] = mul2(g2[e], k1[e]);
            K2[KEEP_K ? 2 * c + e : 0] = k2[e];
          }
#pragma unroll
          for (int i = 0; i < CPT; ++i) {
            f32x2 s = mul2(S.v[i][2 * c + e], g1[e]);
            A1[i] = fma2(s, k1[e], A1[i]);
            B1[i] = fma2(s, q1[e], B1[i]);
            s = mul2(s, g2[e]);
            A2[i] = fma2(s, k2[e], A2[i]);
            B2[i] = fma2(s, q2[e], B2[i]);
            S.v[i][2 * c + e] = s;
          }
        }
      }
      float r[4 * CPT];
#pragma unroll
      for (int i = 0; i < CPT; ++i) {
        const float2 x0 = unpack2(A1[i]), x1 = unpack2(B1[i]), x2 = unpack2(A2[i]), x3 = unpack2(B2[i]);
        r[4 * i] = x0.x + x0.y; r[4 * i + 1] = x1.x + x1.y; r[4 * i + 2] = x2.x + x2.y; r[4 * i + 3] = x3.x + x3.y;
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < 4 * CPT; ++i) r[i] += __shfl_xor_sync(0xffffffffu, r[i], o);
      const float4 s1 = *reinterpret_cast<const float4*>(st + Stage::OFF_S + 4 * t);
      const float4 s2 = *reinterpret_cast<const float4*>(st + Stage::OFF_S + 4 * t + 4);
      float* orow = a.out + (static_cast<int64_t>(t0 + t) * a.heads + w.head) * a.vdim + mycol;
#pragma unroll
      for (int i = 0; i < CPT; ++i) {
        // s1, s2 = (k . q, products with the token before, beta)
        const float v1 = st[Stage::OFF_V + t * COLS + cg * CPT + i], v2 = st[Stage::OFF_V + (t + 1) * COLS + cg * CPT + i];
        const float u1 = s1.w * (v1 - r[4 * i]);
        const float u2 = s2.w * (v2 - fmaf(s2.y, u1, r[4 * i + 2]));
        const f32x2 p1 = pack2(u1, u1), p2 = pack2(u2, u2);
        if (KEEP_K) {
#pragma unroll
          for (int c = 0; c < NCH * 2; ++c) S.v[i][c] = fma2(K2[KEEP_K ? c : 0], p2, fma2(K1[KEEP_K ? c : 0], p1, S.v[i][c]));
        } else {
#pragma unroll
          for (int c = 0; c < NCH; ++c) {
            f32x2 k1[2], k2[2], g2[2];
            lds2(ka + c * 32, k1[0], k1[1]);
            lds2(ka + DP + c * 32, k2[0], k2[1]);
            lds2(ga + DP + c * 32, g2[0], g2[1]);
#pragma unroll
            for (int e = 0; e < 2; ++e) S.v[i][2 * c + e] = fma2(k2[e], p2, fma2(mul2(g2[e], k1[e]), p1, S.v[i][2 * c + e]));
          }
        }
        if (mycol + i < a.vdim) {
          if (l8 == i) orow[i] = fmaf(s1.x, u1, r[4 * i + 1]);
          if (l8 == CPT + i && t + 1 < n) orow[static_cast<int64_t>(a.heads) * a.vdim + i] = fmaf(s2.x, u2, fmaf(s2.z, u1, r[4 * i + 3]));
        }
      }
    }
    __syncthreads();       // the stage may be refilled
  }
  S.store(w.state, mycol, w.columns, l8);
}

// Sums V values per lane over the 16 lanes of a column group, halving the values a lane carries at every exchange:
// lane l of the group returns the total of value l * V / 16.
template <int V>
__device__ __forceinline__ float reduce_scatter16(float (&r)[V], int l16) {
#pragma unroll
  for (int o = 8, cur = V; o > 0; o >>= 1) {
    if (cur > 1) {
      cur >>= 1;
      const bool upper = (l16 & o) != 0;
#pragma unroll
      for (int j = 0; j < cur; ++j) {
        const float send = upper ? r[j] : r[j + cur], keep = upper ? r[j + cur] : r[j];
        r[j] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
    } else {
      r[0] += __shfl_xor_sync(0xffffffffu, r[0], o);
    }
  }
  return r[0];
}

// mLSTM and decay scan, prompt form: sixteen lanes per CPT columns (a shared-memory read costs the same whatever the lanes
// do with it, so a lane's channels serve four columns), sums handed out one per lane.
template <int MODE, int DP, int CPT, int COLS>
__global__ void __launch_bounds__(COLS / CPT * 16) gated_scan_kernel(const mdb_scan_args a) {
  constexpr int NR = DP / 64;            // float4 per lane and column
  using Stage = ScanStage<MODE, DP, COLS>;
  constexpr int TB = Stage::TB, OFF_V = Stage::OFF_V, OFF_S = Stage::OFF_S;
  constexpr int VALS = 2 * CPT, PER = 16 / VALS;      // sums of a pair of tokens; lanes per sum
  extern __shared__ __align__(16) float scan_smem[];
  __shared__ float4 sh_gate[TB];         // forget factor, input factor, exp(-m) per token of the stage
  pdl_launch_dependents();
  pdl_wait();
  const ScanJob w = scan_job<MODE, DP, COLS>(a);
  if (!w.live) return;
  const float skip = MODE == kScanDecay && a.skip != nullptr ? a.skip[w.head] : 0.f;
  const int l16 = threadIdx.x & 15, cg = threadIdx.x >> 4, mycol = w.col0 + cg * CPT;
  f32x2 S[CPT][2 * NR];
#pragma unroll
  for (int i = 0; i < CPT; ++i)
#pragma unroll
    for (int c = 0; c < NR; ++c) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!w.fresh && mycol + i < w.columns)
        x = *reinterpret_cast<const float4*>(w.state + static_cast<int64_t>(mycol + i) * DP + c * 64 + l16 * 4);
      S[i][2 * c] = pack2(x.x, x.y);
      S[i][2 * c + 1] = pack2(x.z, x.w);
    }
  // every block of columns keeps a copy of the running maximum, so that no CTA reads what another writes
  const int blocks = (w.columns + kScanBlockCols - 1) / kScanBlockCols, block0 = w.col0 / kScanBlockCols;
  float* mstate = MODE == kScanMlstm ? a.mstate + (static_cast<int64_t>(w.slot) * a.heads + w.head) * blocks : nullptr;
  float run_max = w.fresh || MODE != kScanMlstm ? 0.f : mstate[block0];
  Stage::fill(a, w, w.t_begin, scan_smem);
  int buf = 0;
  for (int t0 = w.t_begin; t0 < w.t_end; t0 += TB, buf ^= 1) {
    const int n = min(TB, w.t_end - t0);
    Stage::turn(a, w, t0, scan_smem, buf);
    const float* st = scan_smem + buf * Stage::FLOATS;
    // m_t = max(f_t + m_(t-1), i_t) over the stage as a scan of the maps x -> max(x + F, I)
    if (MODE == kScanMlstm && threadIdx.x < 32) {
      const int l = threadIdx.x;
      const float li = l < n ? st[OFF_S + 4 * l] : -INFINITY, lf = l < n ? st[OFF_S + 4 * l + 1] : 0.f;
      float F = lf, I = li;
#pragma unroll
      for (int o = 1; o < TB; o <<= 1) {
        const float Fp = __shfl_up_sync(0xffffffffu, F, o), Ip = __shfl_up_sync(0xffffffffu, I, o);
        if (l >= o) { I = fmaxf(Ip + F, I); F += Fp; }
      }
      const float m = fmaxf(F + run_max, I);
      float mp = __shfl_up_sync(0xffffffffu, m, 1);
      if (l == 0) mp = run_max;
      if (l < n) sh_gate[l] = make_float4(expf(lf + mp - m), expf(li - m), expf(-m), 0.f);
      else if (l < TB) sh_gate[l] = make_float4(1.f, 0.f, 0.f, 0.f);
      run_max = __shfl_sync(0xffffffffu, m, n - 1);
    }
    if (MODE == kScanMlstm) __syncthreads();
    for (int t = 0; t < n; t += 2) {
      const float* k1p = st + t * DP + l16 * 4;
      const float* k2p = k1p + DP;
      // (forget factor, input factor, ...) of the two tokens; the decay scan is handed them
      const float4* gates = MODE == kScanMlstm ? sh_gate : reinterpret_cast<const float4*>(st + OFF_S);
      const float4 ga = gates[t], gb = gates[t + 1];
      const f32x2 f1 = pack2(ga.x, ga.x), f2 = pack2(gb.x, gb.x);
      f32x2 v1[CPT], v2[CPT], acc[CPT][2];
#pragma unroll
      for (int i = 0; i < CPT; ++i) {
        const float y1 = st[OFF_V + t * COLS + cg * CPT + i] * ga.y, y2 = st[OFF_V + (t + 1) * COLS + cg * CPT + i] * gb.y;
        v1[i] = pack2(y1, y1);
        v2[i] = pack2(y2, y2);
        acc[i][0] = acc[i][1] = 0ull;
      }
#pragma unroll
      for (int c = 0; c < NR; ++c) {
        f32x2 k1[2], q1[2], k2[2], q2[2];
        lds2(k1p + c * 64, k1[0], k1[1]);
        lds2(k1p + TB * DP + c * 64, q1[0], q1[1]);
        lds2(k2p + c * 64, k2[0], k2[1]);
        lds2(k2p + TB * DP + c * 64, q2[0], q2[1]);
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int i = 0; i < CPT; ++i) {
            f32x2 s = fma2(k1[e], v1[i], mul2(S[i][2 * c + e], f1));
            acc[i][0] = fma2(s, q1[e], acc[i][0]);
            s = fma2(k2[e], v2[i], mul2(s, f2));
            acc[i][1] = fma2(s, q2[e], acc[i][1]);
            S[i][2 * c + e] = s;
          }
      }
      float r[VALS];
#pragma unroll
      for (int i = 0; i < VALS; ++i) {
        const float2 x = unpack2(acc[i / 2][i % 2]);
        r[i] = x.x + x.y;
      }
      const float sum = reduce_scatter16<VALS>(r, l16);
      const int mine = l16 / PER, col = mine >> 1, kind = mine & 1;      // kind: first or second token of the pair
      if (l16 % PER == 0 && t + kind < n) {
        const int64_t th = static_cast<int64_t>(t0 + t + kind) * a.heads + w.head;
        if (mycol + col < a.vdim)
          a.out[th * a.vdim + mycol + col] = MODE == kScanDecay ? fmaf(skip, st[OFF_V + (t + kind) * COLS + cg * CPT + col], sum) : sum;
        else if (MODE == kScanMlstm && mycol + col == a.vdim) a.den[th] = fmaxf(fabsf(sum), kind ? gb.z : ga.z) + 1e-6f;      // the normaliser's column
      }
    }
    __syncthreads();       // the stage may be refilled
  }
#pragma unroll
  for (int i = 0; i < CPT; ++i)
    if (mycol + i < w.columns) {
#pragma unroll
      for (int c = 0; c < NR; ++c) {
        const float2 lo = unpack2(S[i][2 * c]), hi = unpack2(S[i][2 * c + 1]);
        *reinterpret_cast<float4*>(w.state + static_cast<int64_t>(mycol + i) * DP + c * 64 + l16 * 4) = make_float4(lo.x, lo.y, hi.x, hi.y);
      }
    }
  if (MODE == kScanMlstm && threadIdx.x == 0)
    for (int b = block0; b < blocks && b * kScanBlockCols < w.col0 + COLS; ++b) mstate[b] = run_max;
}

// One-token form: every sequence brings one token and a CTA owns all columns of a head.  The delta rule's decay is computed
// from the raw projection; delta rule and mLSTM normalise and gate the head's output and store it as the next projection's
// input, the decay scan (whose norms span heads) leaves it in fp32.  The state is
// fetched into L2 before the wait for the preceding kernel (a prefetch reads nothing that could be stale).
template <typename T, int MODE, int NCH, int CPT>
__global__ void __launch_bounds__(kScanFusedThreads) scan_token_kernel(const mdb_scan_args a) {
  constexpr int DP = NCH * 32;
  __shared__ __align__(16) float sh[3 * DP];       // k, q, decay
  __shared__ float red[kScanFusedThreads / 32];
  pdl_launch_dependents();
  const int seq = blockIdx.y, head = blockIdx.x;
  const int l8 = threadIdx.x & 7, cg = threadIdx.x >> 3, mycol = cg * CPT;
  const int columns = a.vdim + (MODE == kScanMlstm ? 1 : 0);
  const int slot = a.state_slot[seq];               // a step input, written by no kernel
  const bool ok = slot >= 0 && slot < a.num_slots;
  float* state = a.state + (ok ? slot : 0) * a.state_slot_stride + static_cast<int64_t>(head) * columns * DP;
  if (ok)
    for (int i = threadIdx.x; i < columns * DP / 32; i += blockDim.x)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(state + i * 32));
  pdl_wait();
  if (!ok) {
    if (slot >= a.num_slots && threadIdx.x == 0) report_status(MDB_STATUS_BAD_SLOT);
    return;
  }
  const int64_t t = a.cu_q[seq];
  const bool fresh = a.start[seq] == 0;
  const int kvh = head / (a.heads / a.kv_heads);
  ScanState<NCH, CPT> S;
  S.load(state, mycol, a.vdim, l8, fresh);
  ScanState<MODE == kScanMlstm ? NCH : 1, 1> N;      // the normaliser, in every column group
  float m_old = 0.f;
  const int blocks = (columns + kScanBlockCols - 1) / kScanBlockCols;
  float* mstate = nullptr;
  if constexpr (MODE == kScanMlstm) {
    N.load(state, a.vdim, columns, l8, fresh);
    mstate = a.mstate + (static_cast<int64_t>(slot) * a.heads + head) * blocks;
    if (!fresh) m_old = mstate[0];
  }
  const float s0 = a.s0[t * a.heads + head];
  const float s1 = MODE != kScanDelta ? a.s1[t * a.heads + head] : 0.f;
  float v[CPT];
#pragma unroll
  for (int i = 0; i < CPT; ++i) v[i] = mycol + i < a.vdim ? a.v[(t * a.heads + head) * a.vdim + mycol + i] : 0.f;
  for (int d = threadIdx.x; d < DP; d += blockDim.x) {
    sh[d] = a.k[(t * a.kv_heads + kvh) * DP + d];
    sh[DP + d] = a.q[(t * a.kv_heads + kvh) * DP + d];
    if (MODE == kScanDelta) {
      float r = 1.f;
      if (d < a.dim)
        r = expf(-expf(a.a_log[head]) * softplus_f(rows_at<float>(a.raw_decay, t, head * a.dim + d) + a.dt_bias[head * a.dim + d]));
      sh[2 * DP + d] = r;
    }
  }
  __syncthreads();
  const float* ka = sh + l8 * 4;
  float out[CPT];
  if (MODE == kScanDelta) {
    f32x2 A[CPT], B[CPT], C = 0ull;
#pragma unroll
    for (int i = 0; i < CPT; ++i) A[i] = B[i] = 0ull;
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
      f32x2 k[2], q[2], g[2];
      lds2(ka + c * 32, k[0], k[1]);
      lds2(ka + DP + c * 32, q[0], q[1]);
      lds2(ka + 2 * DP + c * 32, g[0], g[1]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        C = fma2(k[e], q[e], C);
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
          const f32x2 s = mul2(S.v[i][2 * c + e], g[e]);
          A[i] = fma2(s, k[e], A[i]);
          B[i] = fma2(s, q[e], B[i]);
          S.v[i][2 * c + e] = s;
        }
      }
    }
    const float2 cc = unpack2(C);
    const float kq = sum8(cc.x + cc.y);
    f32x2 u2[CPT];
#pragma unroll
    for (int i = 0; i < CPT; ++i) {
      const float2 x = unpack2(A[i]), y = unpack2(B[i]);
      const float u = s0 * (v[i] - sum8(x.x + x.y));
      out[i] = fmaf(kq, u, sum8(y.x + y.y));
      u2[i] = pack2(u, u);
    }
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
      f32x2 k[2];
      lds2(ka + c * 32, k[0], k[1]);
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int i = 0; i < CPT; ++i) S.v[i][2 * c + e] = fma2(k[e], u2[i], S.v[i][2 * c + e]);
    }
  } else {
    const float m_new = fmaxf(s1 + m_old, s0);
    const float fa = MODE == kScanDecay ? s0 : expf(s1 + m_old - m_new), ib = MODE == kScanDecay ? s1 : expf(s0 - m_new);
    const float em = expf(-m_new);
    const f32x2 f2 = pack2(fa, fa), i2 = pack2(ib, ib);
    f32x2 B[CPT], vb[CPT], D = 0ull;
#pragma unroll
    for (int i = 0; i < CPT; ++i) {
      vb[i] = pack2(v[i] * ib, v[i] * ib);
      B[i] = 0ull;
    }
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
      f32x2 k[2], q[2];
      lds2(ka + c * 32, k[0], k[1]);
      lds2(ka + DP + c * 32, q[0], q[1]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
#pragma unroll
        for (int i = 0; i < CPT; ++i) {
          S.v[i][2 * c + e] = fma2(k[e], vb[i], mul2(S.v[i][2 * c + e], f2));
          B[i] = fma2(S.v[i][2 * c + e], q[e], B[i]);
        }
        if constexpr (MODE == kScanMlstm) {
          N.v[0][2 * c + e] = fma2(k[e], i2, mul2(N.v[0][2 * c + e], f2));
          D = fma2(N.v[0][2 * c + e], q[e], D);
        }
      }
    }
    const float2 dd = unpack2(D);
    const float inv = MODE == kScanDecay ? 1.0f : 1.0f / (fmaxf(fabsf(sum8(dd.x + dd.y)), em) + 1e-6f);
#pragma unroll
    for (int i = 0; i < CPT; ++i) {
      const float2 y = unpack2(B[i]);
      out[i] = sum8(y.x + y.y) * inv;
    }
    if constexpr (MODE == kScanMlstm) {
      __syncthreads();             // every column group has read the normaliser and the maximum
      if (cg == 0) N.store(state, a.vdim, columns, l8);
      for (int b = threadIdx.x; b < blocks; b += blockDim.x) mstate[b] = m_new;
    }
  }
  S.store(state, mycol, a.vdim, l8);
  if constexpr (MODE == kScanDecay) {
    const float skip = a.skip != nullptr ? a.skip[head] : 0.f;
#pragma unroll
    for (int i = 0; i < CPT; ++i)
      if (l8 == i && mycol + i < a.vdim) a.out[(t * a.heads + head) * a.vdim + mycol + i] = fmaf(skip, v[i], out[i]);
    return;
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < CPT; ++i)
    if (l8 == i && mycol + i < a.vdim) ss = out[i] * out[i];
  const float rstd = 1.0f / sqrtf(cta_sum(ss, red) / static_cast<float>(a.vdim) + a.eps);
  T* y = static_cast<T*>(a.y) + t * a.ldy + static_cast<int64_t>(head) * a.vdim;
  const float* w = a.norm + static_cast<int64_t>(head) * a.norm_head_stride;
#pragma unroll
  for (int i = 0; i < CPT; ++i)
    if (l8 == i && mycol + i < a.vdim)
      y[mycol + i] = act_from_f<T>(out[i] * rstd * w[mycol + i] * sigmoid_f(rows_at<T>(a.gate, t, head * a.vdim + mycol + i)));
}

}  // namespace mdb

using namespace mdb;

namespace {

// One-token form: at most 64 state registers per thread whatever the key size.
constexpr int scan_token_cols(int dim_pad) { return dim_pad <= 128 ? 4 : 2; }
constexpr int scan_token_groups(int vdim, int cpt) { return ((vdim + cpt - 1) / cpt + 3) / 4 * 4; }

template <typename T, int MODE, int NCH>
int launch_scan_token(const mdb_scan_args& a, cudaStream_t st) {
  if constexpr (NCH * 32 > kScanFusedMaxDim) {
    return MDB_ERR_UNSUPPORTED;
  } else {
    constexpr int CPT = scan_token_cols(NCH * 32);
    const int threads = scan_token_groups(a.vdim, CPT) * 8;
    if (threads > kScanFusedThreads) return MDB_ERR_UNSUPPORTED;
    return mdb_launch(scan_token_kernel<T, MODE, NCH, CPT>, dim3(a.heads, a.bs), dim3(threads), 0, st, a);
  }
}

template <int MODE, int DP, int COLS>
int launch_scan_prompt(const mdb_scan_args& a, cudaStream_t st) {
  constexpr int smem = 2 * ScanStage<MODE, DP, COLS>::FLOATS * 4;
  static_assert(smem <= 227 * 1024, "shared memory of the scan");
  constexpr int DELTA_CPT = DP <= 128 ? 2 : 1, MLSTM_CPT = DP <= 256 ? 4 : 2;
  constexpr int threads = MODE == kScanDelta ? COLS / DELTA_CPT * 8 : COLS / MLSTM_CPT * 16;
  void (*kernel)(mdb_scan_args);
  if constexpr (MODE == kScanDelta) kernel = delta_scan_kernel<DP / 32, DELTA_CPT, COLS>;
  else kernel = gated_scan_kernel<MODE, DP, MLSTM_CPT, COLS>;
  static PerDeviceOnce attr_once;
  const int dev = attr_once.slot();
  if (dev < 0) return MDB_ERR_CUDA;
  if (!attr_once.done[dev]) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return MDB_ERR_CUDA;
    attr_once.done[dev] = true;
  }
  const int columns = a.vdim + (MODE == kScanMlstm ? 1 : 0);
  return mdb_launch(kernel, dim3((columns + COLS - 1) / COLS, a.heads, a.bs), dim3(threads), smem, st, a);
}

template <int MODE, int DP>
int launch_scan_dim(const mdb_scan_args& a, cudaStream_t st) {
  if (a.fused) return a.dtype == MDB_F32 ? launch_scan_token<float, MODE, DP / 32>(a, st) : launch_scan_token<bf16, MODE, DP / 32>(a, st);
  // blocks of 32 columns while they fill the SMs, narrower ones (more re-reads of k, q and g) below that
  const int64_t wide = static_cast<int64_t>((a.vdim + 31) / 32) * a.heads * a.bs;
  return wide >= 148 ? launch_scan_prompt<MODE, DP, 32>(a, st) : launch_scan_prompt<MODE, DP, 16>(a, st);
}

template <int MODE>
int launch_scan(const mdb_scan_args& a, cudaStream_t st) {
  switch (a.dim_pad) {
    case 64: return launch_scan_dim<MODE, 64>(a, st);
    case 128: return launch_scan_dim<MODE, 128>(a, st);
    case 192: return launch_scan_dim<MODE, 192>(a, st);
    case 256: return launch_scan_dim<MODE, 256>(a, st);
    case 512: return launch_scan_dim<MODE, 512>(a, st);
    default: return MDB_ERR_UNSUPPORTED;
  }
}

bool seqs_ok(const int32_t* cu_q, const int32_t* start, const int32_t* slot) { return cu_q && start && slot; }

}  // namespace

extern "C" {

int mdb_scan_dim_pad(int dim) {
  static const int sizes[] = {64, 128, 192, 256, 512};
  for (int s : sizes)
    if (dim <= s) return s;
  return 0;
}

int mdb_scan_blocks(int vdim) { return (vdim + 1 + kScanBlockCols - 1) / kScanBlockCols; }

int mdb_scan_fusable(int dim_pad, int vdim) {
  return dim_pad <= kScanFusedMaxDim && scan_token_groups(vdim, scan_token_cols(dim_pad)) * 8 <= kScanFusedThreads ? 1 : 0;
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
                  seqs_ok(a.cu_q, a.start, a.state_slot) && a.q_out && a.k_out && a.v_out && a.beta_out,
              MDB_ERR_ARG);
  MDB_REQUIRE(a.copy_cols == 0 || (rows_present(a.copy) && a.copy_out && a.copy_cols % 4 == 0 && a.copy_ld % 4 == 0 && rows_ok(a.copy)),
              MDB_ERR_ARG);
  MDB_REQUIRE(a.taps <= kMaxTaps, MDB_ERR_UNSUPPORTED);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int rc;
  if (a.dim % 4 == 0 && a.vdim % 4 == 0 && a.dim <= 128 && a.dim_pad <= 128 && a.taps <= 4 && rows_ok(a.q) && rows_ok(a.k) && rows_ok(a.v) &&
      a.conv_slot_stride % 4 == 0 && mdb_aligned16(a.v_out) && mdb_aligned16(a.conv_q) && mdb_aligned16(a.conv_k) &&
      mdb_aligned16(a.conv_v) && (a.q.parts != nullptr) == (a.k.parts != nullptr) &&
      (a.q.parts != nullptr) == (a.v.parts != nullptr) && (a.copy_cols == 0 || (a.q.parts != nullptr) == (a.copy.parts != nullptr)) &&
      (a.dtype == MDB_BF16 || a.q.parts == nullptr)) {
    const int run = a.m >= 4096 ? 16 : (a.m >= 1024 ? 8 : 1);      // rows a warp walks
    const int units = 2 * a.kv_heads + a.heads * ((a.vdim + 127) / 128) + 1 + (a.copy_cols + 127) / 128;
    // the units of a row tile run next to one another, so that whole rows are read together
    const dim3 grid((units + kPrepWarps - 1) / kPrepWarps, (a.m + run - 1) / run);
    const bool parts = a.q.parts != nullptr;
    const dim3 block(kPrepWarps * 32);
    if (a.dtype == MDB_F32) rc = mdb_launch(delta_prep_rows_kernel<float, false>, grid, block, 0, st, a, run);
    else if (parts) rc = mdb_launch(delta_prep_rows_kernel<bf16, true>, grid, block, 0, st, a, run);
    else rc = mdb_launch(delta_prep_rows_kernel<bf16, false>, grid, block, 0, st, a, run);
  } else {
    const int units = a.kv_heads + a.heads + 1 + (a.copy_cols + 127) / 128;
    const dim3 grid(a.m, (units + kPrepWarps - 1) / kPrepWarps);
    rc = a.dtype == MDB_F32 ? mdb_launch(delta_prep_kernel<float>, grid, dim3(kPrepWarps * 32), 0, st, a)
                            : mdb_launch(delta_prep_kernel<bf16>, grid, dim3(kPrepWarps * 32), 0, st, a);
  }
  if (rc != MDB_OK || a.shift_state || a.taps < 2) return rc;
  const dim3 cgrid((a.channels + 255) / 256, a.bs);
  return a.dtype == MDB_F32 ? mdb_launch(conv_state_kernel<float, mdb_delta_prep_args>, cgrid, dim3(256), 0, st, a)
                            : mdb_launch(conv_state_kernel<bf16, mdb_delta_prep_args>, cgrid, dim3(256), 0, st, a);
}

int mdb_decay_prep(const mdb_decay_prep_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_decay_prep_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.bs >= 0 && a.heads > 0 && a.kv_heads > 0 && a.dim > 0 && a.vdim > 0 && a.taps >= 0, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(a.heads % a.kv_heads == 0 && a.dim_pad >= a.dim && a.dim_pad % 4 == 0, MDB_ERR_ARG);
  MDB_REQUIRE(rows_present(a.q) && rows_present(a.k) && rows_present(a.v), MDB_ERR_ARG);
  MDB_REQUIRE(a.row_seq && seqs_ok(a.cu_q, a.start, a.state_slot) && a.q_out && a.k_out && a.v_out && a.decay_out && a.step_out, MDB_ERR_ARG);
  MDB_REQUIRE(rows_present(a.dt) ? a.a_log && a.dt_bias : a.decay_const != nullptr, MDB_ERR_ARG);
  MDB_REQUIRE(a.taps == 0 || (a.conv && a.conv_bias && (a.conv_state || a.taps == 1)), MDB_ERR_ARG);
  MDB_REQUIRE(a.taps == 0 || a.channels == 2 * a.kv_heads * a.dim + a.heads * a.vdim, MDB_ERR_ARG);
  MDB_REQUIRE(a.taps <= kMaxTaps && (!a.for_chunks || a.dtype == MDB_BF16), MDB_ERR_UNSUPPORTED);
  const bool parts = a.q.parts != nullptr;
  MDB_REQUIRE((a.k.parts != nullptr) == parts && (a.v.parts != nullptr) == parts && (!parts || a.dtype == MDB_BF16), MDB_ERR_UNSUPPORTED);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int rc;
  if (a.dim % 4 == 0 && a.vdim % 4 == 0 && a.taps <= 4 && rows_ok(a.q) && rows_ok(a.k) && rows_ok(a.v) && a.conv_slot_stride % 4 == 0 &&
      mdb_aligned16(a.q_out) && mdb_aligned16(a.k_out) && mdb_aligned16(a.v_out) && mdb_aligned16(a.conv) && mdb_aligned16(a.conv_bias)) {
    const int run = a.m >= 4096 ? 33 : (a.m >= 1024 ? 9 : 1);      // rows a thread walks: one to look the sequence up, then fours
    const int items = a.heads * a.vdim / 4 + 2 * a.kv_heads * (a.dim_pad / 4) + a.heads;
    const dim3 grid((items + kDecayPrepThreads - 1) / kDecayPrepThreads, (a.m + run - 1) / run), block(kDecayPrepThreads);
    MDB_REQUIRE(grid.y <= 65535, MDB_ERR_UNSUPPORTED);
    if (a.dtype == MDB_F32) rc = mdb_launch(decay_prep_rows_kernel<float, float, false>, grid, block, 0, st, a, run);
    else if (a.for_chunks && parts) rc = mdb_launch(decay_prep_rows_kernel<bf16, bf16, true>, grid, block, 0, st, a, run);
    else if (a.for_chunks) rc = mdb_launch(decay_prep_rows_kernel<bf16, bf16, false>, grid, block, 0, st, a, run);
    else if (parts) rc = mdb_launch(decay_prep_rows_kernel<bf16, float, true>, grid, block, 0, st, a, run);
    else rc = mdb_launch(decay_prep_rows_kernel<bf16, float, false>, grid, block, 0, st, a, run);
  } else {
    const int items = a.heads * a.vdim + 2 * a.kv_heads * a.dim_pad + a.heads;
    const dim3 grid(a.m, (items + 255) / 256);
    if (a.dtype == MDB_F32) rc = mdb_launch(decay_prep_kernel<float, float>, grid, dim3(256), 0, st, a);
    else if (a.for_chunks) rc = mdb_launch(decay_prep_kernel<bf16, bf16>, grid, dim3(256), 0, st, a);
    else rc = mdb_launch(decay_prep_kernel<bf16, float>, grid, dim3(256), 0, st, a);
  }
  if (rc != MDB_OK || a.shift_state || a.taps < 2) return rc;
  const dim3 cgrid((a.channels + 255) / 256, a.bs);
  return a.dtype == MDB_F32 ? mdb_launch(conv_state_kernel<float, mdb_decay_prep_args>, cgrid, dim3(256), 0, st, a)
                            : mdb_launch(conv_state_kernel<bf16, mdb_decay_prep_args>, cgrid, dim3(256), 0, st, a);
}

int mdb_channel_decay(const mdb_decay_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_decay_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.dim_pad >= a.dim, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(a.x && a.a_log && a.dt_bias && a.q && a.k && a.g && a.scalars && a.beta && a.row_seq && a.cu_q &&
                  a.ldx >= static_cast<int64_t>(a.heads) * a.dim,
              MDB_ERR_ARG);
  MDB_REQUIRE(a.dim_pad % 4 == 0 && mdb_aligned16(a.g) && mdb_aligned16(a.q) && mdb_aligned16(a.k) && mdb_aligned16(a.scalars), MDB_ERR_ALIGN);
  const dim3 grid(a.m, a.m >= 1024 ? 1 : (a.heads + 3) / 4);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a.dim % 4 == 0 && a.ldx % 4 == 0 && mdb_aligned16(a.x) && mdb_aligned16(a.dt_bias))
    return mdb_launch(channel_decay_kernel<true>, grid, dim3(128), 0, st, a);
  return mdb_launch(channel_decay_kernel<false>, grid, dim3(128), 0, st, a);
}

int mdb_mlstm_prep(const mdb_mlstm_prep_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_mlstm_prep_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.heads > 0 && a.dim > 0 && a.dim_pad >= a.dim && a.vdim > 0 && a.cap > 0.f, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(rows_present(a.q) && rows_present(a.k) && rows_present(a.v) && rows_present(a.i) && rows_present(a.f) &&
                  a.bias_i && a.bias_f && a.q_out && a.k_out && a.v_out && a.log_i && a.log_f,
              MDB_ERR_ARG);
  const int items = a.heads * a.dim_pad / 4 + (a.heads * a.vdim + 3) / 4 + a.heads;
  const dim3 grid(a.m, a.m >= 1024 ? 1 : (items + 255) / 256);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && rows_ok(a.q) && rows_ok(a.k) && rows_ok(a.v) && mdb_aligned16(a.v_out);
  const bool parts = a.q.parts != nullptr;
  if ((a.k.parts != nullptr) != parts || (a.v.parts != nullptr) != parts || (parts && a.dtype == MDB_F32)) return MDB_ERR_UNSUPPORTED;
  if (a.dtype == MDB_F32)
    return vec ? mdb_launch(mlstm_prep_kernel<float, true, false>, grid, dim3(256), 0, st, a)
               : mdb_launch(mlstm_prep_kernel<float, false, false>, grid, dim3(256), 0, st, a);
  if (!vec) return mdb_launch(mlstm_prep_kernel<bf16, false, false>, grid, dim3(256), 0, st, a);
  return parts ? mdb_launch(mlstm_prep_kernel<bf16, true, true>, grid, dim3(256), 0, st, a)
               : mdb_launch(mlstm_prep_kernel<bf16, true, false>, grid, dim3(256), 0, st, a);
}

int mdb_scan(const mdb_scan_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_scan_args a = *args;
  MDB_REQUIRE(a.mode >= MDB_SCAN_DELTA && a.mode <= MDB_SCAN_DECAY, MDB_ERR_ARG);
  MDB_REQUIRE(a.bs >= 0 && a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.vdim > 0, MDB_ERR_ARG);
  if (a.bs == 0) return MDB_OK;
  MDB_REQUIRE(a.q && a.k && a.v && a.state && (a.mode == MDB_SCAN_DELTA ? a.fused == 0 || a.s0 : a.s0 && a.s1) && seqs_ok(a.cu_q, a.start, a.state_slot), MDB_ERR_ARG);
  MDB_REQUIRE(a.mode != MDB_SCAN_MLSTM || (a.mstate && a.kv_heads == a.heads), MDB_ERR_ARG);
  if (a.mode == MDB_SCAN_DECAY) {
    MDB_REQUIRE(a.out != nullptr, MDB_ERR_ARG);
  } else if (a.fused) {
    MDB_REQUIRE(rows_present(a.gate) && a.norm && a.y, MDB_ERR_ARG);
    MDB_REQUIRE(a.mode != MDB_SCAN_DELTA || (rows_present(a.raw_decay) && a.a_log && a.dt_bias), MDB_ERR_ARG);
  } else {
    MDB_REQUIRE(a.out != nullptr && (a.mode == MDB_SCAN_DELTA ? a.g && a.scalars : a.den != nullptr), MDB_ERR_ARG);
  }
  MDB_REQUIRE(mdb_aligned16(a.q) && mdb_aligned16(a.k) && mdb_aligned16(a.g) && mdb_aligned16(a.state) && mdb_aligned16(a.scalars) &&
                  a.state_slot_stride % 4 == 0,
              MDB_ERR_ALIGN);
  MDB_REQUIRE(a.heads <= 65535 && a.bs <= 65535, MDB_ERR_UNSUPPORTED);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a.mode == MDB_SCAN_DECAY) return launch_scan<kScanDecay>(a, st);
  return a.mode == MDB_SCAN_DELTA ? launch_scan<kScanDelta>(a, st) : launch_scan<kScanMlstm>(a, st);
}

}  // extern "C"
