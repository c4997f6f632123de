// Row kernels of the decoders whose residual stream is kept in fp32: embedding with a scale, residual add (from a
// projection, from split-k slices, from the outputs of a mixture of experts) fused with the RMSNorm that follows,
// RMSNorm of column segments of a projection (one of which may go straight into a paged cache), the per-head
// normalisation and output gate behind a recurrence, and the row gather out of a paged latent cache.
// Activations are bf16 or fp32 (template parameter), all arithmetic is fp32.
#include "mdb_common.cuh"

namespace mdb {

template <typename T> __device__ __forceinline__ float act_to_f(T v);
template <> __device__ __forceinline__ float act_to_f<bf16>(bf16 v) { return __bfloat162float(v); }
template <> __device__ __forceinline__ float act_to_f<float>(float v) { return v; }
template <typename T> __device__ __forceinline__ T act_from_f(float v);
template <> __device__ __forceinline__ bf16 act_from_f<bf16>(float v) { return __float2bfloat16_rn(v); }
template <> __device__ __forceinline__ float act_from_f<float>(float v) { return v; }

template <typename T> __device__ __forceinline__ float4 act_load4(const T* p);
template <> __device__ __forceinline__ float4 act_load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 act_load4<bf16>(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T> __device__ __forceinline__ void act_store4(T* p, float4 v);
template <> __device__ __forceinline__ void act_store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void act_store4<bf16>(bf16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// A projection's output as its consumer finds it: rows of T, or fp32 split-k slices that the consumer sums in slice
// order and rounds to T, as the projection itself would have.
template <typename T>
__device__ __forceinline__ float rows_at(const mdb_rows& s, int64_t row, int col) {
  const int64_t off = row * s.ld + s.col + col;
  if (s.parts != nullptr) {
    float a = 0.f;
    for (int p = 0; p < s.nparts; ++p) a += s.parts[p * s.part_stride + off];
    return act_to_f(act_from_f<T>(a));
  }
  return act_to_f(static_cast<const T*>(s.x)[off]);
}
template <typename T>
__device__ __forceinline__ float4 rows_at4(const mdb_rows& s, int64_t row, int col) {
  const int64_t off = row * s.ld + s.col + col;
  if (s.parts != nullptr) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int p0 = 0; p0 < s.nparts; p0 += 8) {
      float4 v[8];                       // eight slices requested together: one round trip to L2 instead of eight
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (p0 + i < s.nparts) v[i] = *reinterpret_cast<const float4*>(s.parts + (p0 + i) * s.part_stride + off);
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (p0 + i < s.nparts) { a.x += v[i].x; a.y += v[i].y; a.z += v[i].z; a.w += v[i].w; }
    }
    a.x = act_to_f(act_from_f<T>(a.x)); a.y = act_to_f(act_from_f<T>(a.y));
    a.z = act_to_f(act_from_f<T>(a.z)); a.w = act_to_f(act_from_f<T>(a.w));
    return a;
  }
  return act_load4(static_cast<const T*>(s.x) + off);
}
// The form known at compile time: kernels that read many places keep the slice loop out of their row form.
template <typename T, bool PARTS>
__device__ __forceinline__ float4 rows_at4_of(const mdb_rows& s, int64_t row, int col) {
  const int64_t off = row * s.ld + s.col + col;
  if (!PARTS) return act_load4(static_cast<const T*>(s.x) + off);
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
  for (int p = 0; p < s.nparts; ++p) {
    const float4 v = *reinterpret_cast<const float4*>(s.parts + p * s.part_stride + off);
    a.x += v.x; a.y += v.y; a.z += v.z; a.w += v.w;
  }
  return make_float4(act_to_f(act_from_f<T>(a.x)), act_to_f(act_from_f<T>(a.y)), act_to_f(act_from_f<T>(a.z)), act_to_f(act_from_f<T>(a.w)));
}
__host__ __device__ __forceinline__ bool rows_present(const mdb_rows& s) { return s.x != nullptr || s.parts != nullptr; }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

// Sum over the CTA; `red` holds one float per warp and is free again after the call's last barrier.
__device__ __forceinline__ float cta_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < static_cast<int>(blockDim.x + 31) / 32; ++w) t += red[w];
  return t;
}

constexpr int kRes32Threads = 256;

// One CTA per row.  residual (scaled or, with ids, = embed[id] * scale) + up to two projections + the weighted sum of
// the chosen experts' rows; y = residual / rms * weight.  POST: the norm replaces the residual, and y is the new residual or
// its norm with a second weight.  NV float4 chunks of the row per thread; PARTS: a projection may come as split-k slices.
template <typename T, int NV, bool POST, bool PARTS>
__global__ void __launch_bounds__(kRes32Threads) residual_norm_kernel(const mdb_residual_norm_args a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[kRes32Threads / 32];
  const int64_t row = blockIdx.x;
  float* res = a.residual + row * a.width_pad;
  float4 v[NV];
  float ss = 0.f;
  int64_t id = 0;
  if (a.ids != nullptr) {
    id = a.ids[row];
    if (id < 0 || id >= a.vocab) {
      if (threadIdx.x == 0) report_status(MDB_STATUS_BAD_TOKEN);
      id = -1;
    }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * kRes32Threads) * 4;
    if (c >= a.width_pad) continue;
    float4 x;
    if (a.ids != nullptr) {
      x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (id >= 0) {
        x = act_load4(static_cast<const T*>(a.embed) + id * a.width_pad + c);
        x.x *= a.embed_scale; x.y *= a.embed_scale; x.z *= a.embed_scale; x.w *= a.embed_scale;
      }
    } else {
      x = *reinterpret_cast<const float4*>(res + c);
      if (POST) { x.x *= a.res_scale; x.y *= a.res_scale; x.z *= a.res_scale; x.w *= a.res_scale; }
    }
#pragma unroll
    for (int s = 0; s < 2; ++s) {
      if (!rows_present(a.add[s])) continue;
      const float4 d = PARTS ? rows_at4<T>(a.add[s], row, c) : rows_at4_of<T, false>(a.add[s], row, c);
      x.x += d.x; x.y += d.y; x.z += d.z; x.w += d.w;
    }
    if (a.moe_rows != nullptr) {
      float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int k = 0; k < a.moe_top; ++k) {
        const int slot = a.moe_slot[row * a.moe_top + k];
        if (slot < 0) continue;
        const float w = a.moe_weight[row * a.moe_top + k];
        const float4 e = act_load4(static_cast<const T*>(a.moe_rows) + slot * a.moe_ld + c);
        d.x = fmaf(w, e.x, d.x); d.y = fmaf(w, e.y, d.y); d.z = fmaf(w, e.z, d.z); d.w = fmaf(w, e.w, d.w);
      }
      x.x += d.x; x.y += d.y; x.z += d.z; x.w += d.w;
    }
    if (!POST) *reinterpret_cast<float4*>(res + c) = x;
    v[i] = x;
    ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;      // columns past width hold zeros
  }
  if (!POST && a.y == nullptr) return;
  T* y = static_cast<T*>(a.y) + row * a.ldy;
  if (!POST && a.weight == nullptr) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * kRes32Threads) * 4;
      if (c < a.width_pad) act_store4(y + c, v[i]);
    }
    return;
  }
  float rstd = 1.0f / sqrtf(cta_sum(ss, red) / static_cast<float>(a.width) + a.eps);
  if (POST) {
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (threadIdx.x + i * kRes32Threads) * 4;
      if (c >= a.width_pad) continue;
      const float4 w = *reinterpret_cast<const float4*>(a.weight + c);
      v[i] = make_float4(v[i].x * rstd * w.x, v[i].y * rstd * w.y, v[i].z * rstd * w.z, v[i].w * rstd * w.w);
      *reinterpret_cast<float4*>(res + c) = v[i];
      if (a.y != nullptr && a.weight2 == nullptr) act_store4(y + c, v[i]);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    if (a.y == nullptr || a.weight2 == nullptr) return;
    rstd = 1.0f / sqrtf(cta_sum(ss, red) / static_cast<float>(a.width) + a.eps);
  }
  const float* weight = POST ? a.weight2 : a.weight;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * kRes32Threads) * 4;
    if (c >= a.width_pad) continue;
    const float4 w = *reinterpret_cast<const float4*>(weight + c);
    act_store4(y + c, make_float4(v[i].x * rstd * w.x, v[i].y * rstd * w.y, v[i].z * rstd * w.z, v[i].w * rstd * w.w));
  }
}

// One CTA per (row, segment): RMSNorm of n columns of a projection, zero-padded to n_pad, into row `row` of the
// output or, with slots, into cache row slots[row].
struct RmsSegments {
  mdb_rms_segment s[MDB_MAX_RMS_SEGMENTS];
};
constexpr int kRmsRowsThreads = 128;
template <typename T, bool PARTS>
__global__ void __launch_bounds__(kRmsRowsThreads) rms_rows_kernel(const RmsSegments segs) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[kRmsRowsThreads / 32];
  const mdb_rms_segment& s = segs.s[blockIdx.y];
  const int64_t row = blockIdx.x;
  int64_t out_row = row;
  if (s.slots != nullptr) {
    const int slot = s.slots[row];
    if (slot == -1) return;
    if (slot < 0 || slot >= s.num_slots) {
      if (threadIdx.x == 0) report_status(MDB_STATUS_BAD_SLOT);
      return;
    }
    out_row = slot;
  }
  T* out = static_cast<T*>(s.out) + out_row * s.ld_out;
  // columns n .. n_pad of the projection are zeros; the first kKeep pieces of the row stay in registers
  constexpr int kKeep = 4;
  float4 v[kKeep];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = (threadIdx.x + i * kRmsRowsThreads) * 4;
    v[i] = c < s.n_pad ? rows_at4_of<T, PARTS>(s.src, row, c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int i = 0; i < kKeep; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
  for (int c = (threadIdx.x + kKeep * kRmsRowsThreads) * 4; c < s.n_pad; c += kRmsRowsThreads * 4) {
    const float4 x = rows_at4_of<T, PARTS>(s.src, row, c);
    ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
  }
  const float rstd = 1.0f / sqrtf(cta_sum(ss, red) / static_cast<float>(s.n) + s.eps);
  auto put = [&](int c, float4 x) {
    const float4 w = *reinterpret_cast<const float4*>(s.weight + c);
    act_store4(out + c, make_float4(x.x * rstd * w.x, x.y * rstd * w.y, x.z * rstd * w.z, x.w * rstd * w.w));
  };
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = (threadIdx.x + i * kRmsRowsThreads) * 4;
    if (c < s.n_pad) put(c, v[i]);
  }
  for (int c = (threadIdx.x + kKeep * kRmsRowsThreads) * 4; c < s.n_pad; c += kRmsRowsThreads * 4)
    put(c, rows_at4_of<T, PARTS>(s.src, row, c));
}

// Behind a recurrence: a warp per (row, head).  y = o' / rms(o') * weight * sigmoid(gate), o' = o / den where there is
// a den.  VEC: heads in multiples of four, everything 16-byte aligned; up to 256 values stay in registers between the
// two passes, and the gate is requested with them.
template <typename T, bool VEC, bool PARTS>
__global__ void __launch_bounds__(128) gated_norm_kernel(const mdb_gated_norm_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int lane = threadIdx.x & 31;
  constexpr int kKeep = 2;
#pragma unroll 2
  for (int head = blockIdx.y * 4 + (threadIdx.x >> 5); head < a.heads; head += gridDim.y * 4) {
    const float* o = a.o + (row * a.heads + head) * a.vdim;
    const float den = a.den != nullptr ? a.den[row * a.heads + head] : 1.0f;
    const float* w = a.weight + static_cast<int64_t>(head) * a.weight_head_stride;
    T* y = static_cast<T*>(a.y) + row * a.ldy + static_cast<int64_t>(head) * a.vdim;
    float ss = 0.f;
    if (VEC) {
      float4 v[kKeep], g[kKeep];
#pragma unroll
      for (int i = 0; i < kKeep; ++i) {
        const int c = lane * 4 + 128 * i;
        v[i] = g[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < a.vdim) {
          v[i] = *reinterpret_cast<const float4*>(o + c);
          g[i] = rows_at4_of<T, PARTS>(a.gate, row, head * a.vdim + c);
        }
        ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
      }
      for (int c = lane * 4 + 128 * kKeep; c < a.vdim; c += 128) {
        const float4 x = *reinterpret_cast<const float4*>(o + c);
        ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
      }
      const float inv = 1.0f / den, rstd = inv / sqrtf(warp_sum(ss) * inv * inv / static_cast<float>(a.vdim) + a.eps);
      auto put = [&](int c, float4 x, float4 gv) {
        const float4 wv = *reinterpret_cast<const float4*>(w + c);
        act_store4(y + c, make_float4(x.x * rstd * wv.x * sigmoid_f(gv.x), x.y * rstd * wv.y * sigmoid_f(gv.y),
                                      x.z * rstd * wv.z * sigmoid_f(gv.z), x.w * rstd * wv.w * sigmoid_f(gv.w)));
      };
#pragma unroll
      for (int i = 0; i < kKeep; ++i)
        if (lane * 4 + 128 * i < a.vdim) put(lane * 4 + 128 * i, v[i], g[i]);
      for (int c = lane * 4 + 128 * kKeep; c < a.vdim; c += 128)
        put(c, *reinterpret_cast<const float4*>(o + c), rows_at4_of<T, PARTS>(a.gate, row, head * a.vdim + c));
    } else {
      for (int c = lane; c < a.vdim; c += 32) ss += o[c] * o[c];
      const float inv = 1.0f / den, rstd = inv / sqrtf(warp_sum(ss) * inv * inv / static_cast<float>(a.vdim) + a.eps);
      for (int c = lane; c < a.vdim; c += 32)
        y[c] = act_from_f<T>(o[c] * rstd * w[c] * sigmoid_f(rows_at<T>(a.gate, row, head * a.vdim + c)));
    }
  }
}

// A CTA per (row, part): one root mean square over the part's columns of a row, gate before the norm (silu) or after the weight
// (sigmoid).  The first kKeep pieces stay in registers between the two passes.
constexpr int kPartNormThreads = 256;
template <typename T, bool VEC, bool PARTS>
__global__ void __launch_bounds__(kPartNormThreads) part_norm_kernel(const mdb_part_norm_args a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[kPartNormThreads / 32];
  const int64_t row = blockIdx.x;
  const int n = a.n / a.parts, col0 = blockIdx.y * n;
  const float* o = a.o + row * a.n + col0;
  const float* w = a.weight + col0;
  T* y = static_cast<T*>(a.y) + row * a.ldy + col0;
  if (VEC) {
    constexpr int kKeep = 4;
    const int step = blockDim.x * 4;
    float4 v[kKeep], g[kKeep];
    auto gated = [&](float4 x, float4 z) {
      return a.gate_first ? make_float4(x.x * z.x * sigmoid_f(z.x), x.y * z.y * sigmoid_f(z.y), x.z * z.z * sigmoid_f(z.z), x.w * z.w * sigmoid_f(z.w)) : x;
    };
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int c = threadIdx.x * 4 + i * step;
      v[i] = g[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < n) {
        v[i] = *reinterpret_cast<const float4*>(o + c);
        g[i] = rows_at4_of<T, PARTS>(a.gate, row, col0 + c);
      }
    }
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      v[i] = gated(v[i], g[i]);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    for (int c = threadIdx.x * 4 + kKeep * step; c < n; c += step) {
      const float4 x = gated(*reinterpret_cast<const float4*>(o + c), rows_at4_of<T, PARTS>(a.gate, row, col0 + c));
      ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    }
    const float rstd = a.out_scale / sqrtf(cta_sum(ss, red) / static_cast<float>(n) + a.eps);
    auto put = [&](int c, float4 x, float4 z) {
      const float4 wv = *reinterpret_cast<const float4*>(w + c);
      x = make_float4(x.x * rstd * wv.x, x.y * rstd * wv.y, x.z * rstd * wv.z, x.w * rstd * wv.w);
      if (!a.gate_first) x = make_float4(x.x * sigmoid_f(z.x), x.y * sigmoid_f(z.y), x.z * sigmoid_f(z.z), x.w * sigmoid_f(z.w));
      act_store4(y + c, x);
    };
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int c = threadIdx.x * 4 + i * step;
      if (c < n) put(c, v[i], g[i]);
    }
    for (int c = threadIdx.x * 4 + kKeep * step; c < n; c += step) {
      const float4 z = rows_at4_of<T, PARTS>(a.gate, row, col0 + c);
      put(c, gated(*reinterpret_cast<const float4*>(o + c), z), z);
    }
  } else {
    auto value = [&](int c, float z) { return a.gate_first ? o[c] * z * sigmoid_f(z) : o[c]; };
    float ss = 0.f;
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
      const float x = value(c, rows_at<T>(a.gate, row, col0 + c));
      ss += x * x;
    }
    const float rstd = a.out_scale / sqrtf(cta_sum(ss, red) / static_cast<float>(n) + a.eps);
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
      const float z = rows_at<T>(a.gate, row, col0 + c);
      y[c] = act_from_f<T>(value(c, z) * rstd * w[c] * (a.gate_first ? 1.0f : sigmoid_f(z)));
    }
  }
}

// The same for parts of at most 1024 columns: a warp per (row, part), everything in registers, no barrier.
template <typename T, int NK, bool PARTS>
__global__ void __launch_bounds__(kPartNormThreads) part_norm_warp_kernel(const mdb_part_norm_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * (kPartNormThreads / 32) + (threadIdx.x >> 5);
  const int64_t row = unit / a.parts;
  if (row >= a.m) return;
  const int n = a.n / a.parts, col0 = static_cast<int>(unit % a.parts) * n, lane = threadIdx.x & 31;
  const float* o = a.o + row * a.n + col0;
  float4 v[NK], g[NK];
#pragma unroll
  for (int i = 0; i < NK; ++i) {
    const int c = lane * 4 + 128 * i;
    v[i] = g[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < n) {
      v[i] = *reinterpret_cast<const float4*>(o + c);
      g[i] = rows_at4_of<T, PARTS>(a.gate, row, col0 + c);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NK; ++i) {
    const float4 s = make_float4(sigmoid_f(g[i].x), sigmoid_f(g[i].y), sigmoid_f(g[i].z), sigmoid_f(g[i].w));
    if (a.gate_first) v[i] = make_float4(v[i].x * g[i].x * s.x, v[i].y * g[i].y * s.y, v[i].z * g[i].z * s.z, v[i].w * g[i].w * s.w);
    ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    g[i] = a.gate_first ? make_float4(1.f, 1.f, 1.f, 1.f) : s;
  }
  const float rstd = a.out_scale / sqrtf(warp_sum(ss) / static_cast<float>(n) + a.eps);
  T* y = static_cast<T*>(a.y) + row * a.ldy + col0;
#pragma unroll
  for (int i = 0; i < NK; ++i) {
    const int c = lane * 4 + 128 * i;
    if (c >= n) continue;
    const float4 w = *reinterpret_cast<const float4*>(a.weight + col0 + c);
    act_store4(y + c, make_float4(v[i].x * rstd * w.x * g[i].x, v[i].y * rstd * w.y * g[i].y, v[i].z * rstd * w.z * g[i].z, v[i].w * rstd * w.w * g[i].w));
  }
}

template <typename T, bool PARTS>
static int launch_part_norm_warp(const mdb_part_norm_args& a, cudaStream_t st) {
  const int n = a.n / a.parts;
  const int64_t units = static_cast<int64_t>(a.m) * a.parts;
  const dim3 grid(static_cast<unsigned>((units + kPartNormThreads / 32 - 1) / (kPartNormThreads / 32))), block(kPartNormThreads);
  if (n <= 128) return mdb_launch(part_norm_warp_kernel<T, 1, PARTS>, grid, block, 0, st, a);
  if (n <= 256) return mdb_launch(part_norm_warp_kernel<T, 2, PARTS>, grid, block, 0, st, a);
  if (n <= 512) return mdb_launch(part_norm_warp_kernel<T, 4, PARTS>, grid, block, 0, st, a);
  return mdb_launch(part_norm_warp_kernel<T, 8, PARTS>, grid, block, 0, st, a);
}

// Row r of the output = the latent of token r - cu[seq] of its sequence, read through the page table.
template <typename T>
__global__ void __launch_bounds__(64) gather_latents_kernel(const T* cache, const int32_t* table,
                                                            int table_stride, int num_pages, const int32_t* cu,
                                                            int nseq, T* out, int width) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x;
  int lo = 0, hi = nseq;                         // the last sequence that starts at or before this row
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (cu[mid] <= row) lo = mid; else hi = mid;
  }
  const int pos = row - cu[lo];
  int page = pos / kPage < table_stride ? table[static_cast<int64_t>(lo) * table_stride + pos / kPage] : -1;
  if (page < 0 || page >= num_pages) {
    if (threadIdx.x == 0) report_status(MDB_STATUS_BAD_PAGE);
    page = 0;
  }
  const uint4* src = reinterpret_cast<const uint4*>(cache + (static_cast<int64_t>(page) * kPage + pos % kPage) * width);
  uint4* dst = reinterpret_cast<uint4*>(out + static_cast<int64_t>(row) * width);
  const int chunks = width * static_cast<int>(sizeof(T)) / 16;
  for (int c = threadIdx.x; c < chunks; c += 64) dst[c] = src[c];
}

// Last kernel of a causal step: one CTA per wanted row of fp32 logits.  token = argmax of logit / temperature +
// Gumbel noise, or of the logit itself where the row asks for the greedy choice (temperature 0); ties go to the
// lower id.
constexpr int kPickThreads = 512;
__global__ void __launch_bounds__(kPickThreads)
pick_token_kernel(const float* logits, int64_t ld, int vocab, const float* temperatures,
                  uint32_t seed, const uint32_t* step_dev, int64_t* out,
                  uint32_t* status_out) {
  pdl_launch_dependents();
  pdl_wait();
  if (status_out != nullptr && blockIdx.x == 0 && threadIdx.x == 0) *status_out = atomicExch(&g_device_status, 0u);
  __shared__ float sv[kPickThreads / 32];
  __shared__ int si[kPickThreads / 32];
  const int row = blockIdx.x;
  const float temp = temperatures[row];
  const float inv = temp > 0.f ? 1.0f / temp : 1.0f;
  const uint32_t key = gumbel_row_key(seed, step_dev != nullptr ? *step_dev : 0u, row);
  float bv = -INFINITY;
  int bi = 0x7fffffff;
  for (int c = threadIdx.x; c < vocab; c += kPickThreads) {
    float v = logits[row * ld + c] * inv;
    if (temp > 0.f) v += gumbel_from_key(key, c);
    if (v > bv) { bv = v; bi = c; }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
  }
  if ((threadIdx.x & 31) == 0) { sv[threadIdx.x >> 5] = bv; si[threadIdx.x >> 5] = bi; }
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int w = 1; w < kPickThreads / 32; ++w)
      if (sv[w] > bv || (sv[w] == bv && si[w] < bi)) { bv = sv[w]; bi = si[w]; }
    out[row] = bi == 0x7fffffff ? 0 : bi;
  }
}

}  // namespace mdb

using namespace mdb;

namespace {
bool rows_ok(const mdb_rows& s) {
  return !rows_present(s) || (s.ld % 4 == 0 && s.col % 4 == 0 && mdb_aligned16(s.x) && mdb_aligned16(s.parts) &&
                              (s.parts == nullptr || (s.nparts >= 1 && s.part_stride % 4 == 0)));
}

template <typename T, bool POST, bool PARTS>
int launch_residual_norm_of(const mdb_residual_norm_args& a, cudaStream_t st) {
  const int chunks = (a.width_pad / 4 + kRes32Threads - 1) / kRes32Threads;
  if (chunks <= 1) return mdb_launch(residual_norm_kernel<T, 1, POST, PARTS>, dim3(a.m), dim3(kRes32Threads), 0, st, a);
  if (chunks <= 2) return mdb_launch(residual_norm_kernel<T, 2, POST, PARTS>, dim3(a.m), dim3(kRes32Threads), 0, st, a);
  if (chunks <= 4) return mdb_launch(residual_norm_kernel<T, 4, POST, PARTS>, dim3(a.m), dim3(kRes32Threads), 0, st, a);
  if (chunks <= 8) return mdb_launch(residual_norm_kernel<T, 8, POST, PARTS>, dim3(a.m), dim3(kRes32Threads), 0, st, a);
  return MDB_ERR_UNSUPPORTED;
}
template <typename T, bool POST>
int launch_residual_norm(const mdb_residual_norm_args& a, cudaStream_t st) {
  return a.add[0].parts != nullptr || a.add[1].parts != nullptr ? launch_residual_norm_of<T, POST, true>(a, st)
                                                                : launch_residual_norm_of<T, POST, false>(a, st);
}
}  // namespace

extern "C" {

int mdb_residual_norm(const mdb_residual_norm_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_residual_norm_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.width > 0 && a.width_pad >= a.width, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(a.residual && (a.ids == nullptr || (a.embed && a.vocab > 0)), MDB_ERR_ARG);
  MDB_REQUIRE(a.y == nullptr || (a.ldy >= a.width_pad && a.ldy % 4 == 0), MDB_ERR_ARG);
  MDB_REQUIRE(a.post ? a.weight != nullptr && a.ids == nullptr : a.weight2 == nullptr && a.res_scale == 1.0f, MDB_ERR_ARG);
  MDB_REQUIRE(a.moe_rows == nullptr || (a.moe_slot && a.moe_weight && a.moe_top > 0 && a.moe_ld % 4 == 0), MDB_ERR_ARG);
  MDB_REQUIRE(a.width_pad % 4 == 0 && rows_ok(a.add[0]) && rows_ok(a.add[1]) && mdb_aligned16(a.residual) &&
                  mdb_aligned16(a.embed) && mdb_aligned16(a.weight) && mdb_aligned16(a.weight2) && mdb_aligned16(a.y) &&
                  mdb_aligned16(a.moe_rows),
              MDB_ERR_ALIGN);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a.post) return a.dtype == MDB_F32 ? launch_residual_norm<float, true>(a, st) : launch_residual_norm<bf16, true>(a, st);
  return a.dtype == MDB_F32 ? launch_residual_norm<float, false>(a, st) : launch_residual_norm<bf16, false>(a, st);
}

int mdb_rms_rows(int dtype, const mdb_rms_segment* segments, int nseg, int m, mdb_stream_t stream) {
  MDB_REQUIRE(segments && nseg >= 1 && nseg <= MDB_MAX_RMS_SEGMENTS && m >= 0, MDB_ERR_ARG);
  if (m == 0) return MDB_OK;
  RmsSegments segs = {};
  for (int i = 0; i < nseg; ++i) {
    const mdb_rms_segment& s = segments[i];
    MDB_REQUIRE(s.n > 0 && s.n_pad >= s.n && s.weight && s.out && s.ld_out >= s.n_pad && rows_present(s.src), MDB_ERR_ARG);
    MDB_REQUIRE(s.n_pad % 4 == 0 && s.ld_out % 4 == 0 && rows_ok(s.src) && mdb_aligned16(s.weight) && mdb_aligned16(s.out),
                MDB_ERR_ALIGN);
    segs.s[i] = s;
  }
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool parts = segs.s[0].src.parts != nullptr;
  for (int i = 1; i < nseg; ++i) MDB_REQUIRE((segs.s[i].src.parts != nullptr) == parts, MDB_ERR_UNSUPPORTED);
  const dim3 grid(m, nseg), block(kRmsRowsThreads);
  if (dtype == MDB_F32)
    return parts ? mdb_launch(rms_rows_kernel<float, true>, grid, block, 0, st, segs) : mdb_launch(rms_rows_kernel<float, false>, grid, block, 0, st, segs);
  return parts ? mdb_launch(rms_rows_kernel<bf16, true>, grid, block, 0, st, segs) : mdb_launch(rms_rows_kernel<bf16, false>, grid, block, 0, st, segs);
}

int mdb_gated_norm(const mdb_gated_norm_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_gated_norm_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.heads > 0 && a.vdim > 0, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(a.o && a.weight && a.y && rows_present(a.gate) && a.ldy >= static_cast<int64_t>(a.heads) * a.vdim, MDB_ERR_ARG);
  // many rows: a CTA takes all heads of its row
  const dim3 grid(a.m, a.m >= 1024 ? 1 : (a.heads + 3) / 4);
  const bool vec = a.vdim % 4 == 0 && rows_ok(a.gate) && a.ldy % 4 == 0 && mdb_aligned16(a.o) && mdb_aligned16(a.y) &&
                   mdb_aligned16(a.weight) && a.weight_head_stride % 4 == 0;
  const bool parts = a.gate.parts != nullptr;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a.dtype == MDB_F32)
    return vec && !parts ? mdb_launch(gated_norm_kernel<float, true, false>, grid, dim3(128), 0, st, a)
                         : mdb_launch(gated_norm_kernel<float, false, true>, grid, dim3(128), 0, st, a);
  if (!vec) return mdb_launch(gated_norm_kernel<bf16, false, true>, grid, dim3(128), 0, st, a);
  return parts ? mdb_launch(gated_norm_kernel<bf16, true, true>, grid, dim3(128), 0, st, a)
               : mdb_launch(gated_norm_kernel<bf16, true, false>, grid, dim3(128), 0, st, a);
}

int mdb_part_norm(const mdb_part_norm_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_part_norm_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.n > 0 && a.parts > 0 && a.n % a.parts == 0, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(a.o && a.weight && a.y && rows_present(a.gate) && a.ldy >= a.n, MDB_ERR_ARG);
  MDB_REQUIRE(a.parts <= 65535, MDB_ERR_UNSUPPORTED);
  const int n = a.n / a.parts;
  const bool vec = n % 4 == 0 && rows_ok(a.gate) && a.ldy % 4 == 0 && mdb_aligned16(a.o) && mdb_aligned16(a.y) && mdb_aligned16(a.weight);
  const bool parts = a.gate.parts != nullptr;
  const dim3 grid(a.m, a.parts), block(n <= 2048 ? 128 : kPartNormThreads);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (vec && n <= 1024 && !(parts && a.dtype == MDB_F32)) {
    if (a.dtype == MDB_F32) return launch_part_norm_warp<float, false>(a, st);
    return parts ? launch_part_norm_warp<bf16, true>(a, st) : launch_part_norm_warp<bf16, false>(a, st);
  }
  if (a.dtype == MDB_F32)
    return vec && !parts ? mdb_launch(part_norm_kernel<float, true, false>, grid, block, 0, st, a)
                         : mdb_launch(part_norm_kernel<float, false, true>, grid, block, 0, st, a);
  if (!vec) return mdb_launch(part_norm_kernel<bf16, false, true>, grid, block, 0, st, a);
  return parts ? mdb_launch(part_norm_kernel<bf16, true, true>, grid, block, 0, st, a)
               : mdb_launch(part_norm_kernel<bf16, true, false>, grid, block, 0, st, a);
}

int mdb_gather_latents(int dtype, const void* cache, const int32_t* block_table, int table_stride, int num_pages,
                       const int32_t* cu, int nseq, int total, void* out, int width, mdb_stream_t stream) {
  MDB_REQUIRE(total >= 0 && nseq >= 0 && width > 0 && num_pages > 0 && table_stride > 0, MDB_ERR_ARG);
  if (total == 0 || nseq == 0) return MDB_OK;
  MDB_REQUIRE(cache && block_table && cu && out, MDB_ERR_ARG);
  MDB_REQUIRE(width % 8 == 0 && mdb_aligned16(cache) && mdb_aligned16(out), MDB_ERR_ALIGN);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == MDB_F32)
    return mdb_launch(gather_latents_kernel<float>, dim3(total), dim3(64), 0, st, static_cast<const float*>(cache),
                      block_table, table_stride, num_pages, cu, nseq, static_cast<float*>(out), width);
  return mdb_launch(gather_latents_kernel<bf16>, dim3(total), dim3(64), 0, st, static_cast<const bf16*>(cache), block_table,
                    table_stride, num_pages, cu, nseq, static_cast<bf16*>(out), width);
}

int mdb_pick_token(const float* logits, int64_t ld, int m, int vocab, const float* temperatures, uint32_t seed,
                   const uint32_t* step_dev, int64_t* out, uint32_t* status_out, mdb_stream_t stream) {
  MDB_REQUIRE(m >= 0 && vocab > 0 && ld >= vocab, MDB_ERR_ARG);
  if (m == 0) return MDB_OK;
  MDB_REQUIRE(logits && temperatures && out, MDB_ERR_ARG);
  return mdb_launch(pick_token_kernel, dim3(m), dim3(kPickThreads), 0, static_cast<cudaStream_t>(stream), logits, ld, vocab,
                    temperatures, seed, step_dev, out, status_out);
}

}  // extern "C"
