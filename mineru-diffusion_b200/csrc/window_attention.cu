// Rotary grouped-query attention over paged K and V caches, with a window and a sink: the kernel in front of it (per-head
// norms, rotation, cache rows) and the forms that take a few tokens of a sequence, decoding above all.  Prompt portions
// go to the window form of the tensor-memory kernel (attention_tc.cu).
//
//   rotary_commit_kernel     a CTA per token: sines and cosines once, then a warp per head.
//   window_attn_mma_kernel   bf16: a CTA takes up to 16 query heads of one KV head of one token and a range of its keys (split
//                            over CTAs, merged by window_combine_kernel).  Its four warps are independent until the end:
//                            each takes every fourth tile of 16 keys through a cp.async ring of its own, with m16n8k16
//                            products whose 16 rows are the heads, and its own running maximum and sum.  A 128-row
//                            tile of the tensor-memory kind would be seven-eighths empty.  Softmax in fp32; the weights enter
//                            the second product as the sum of two bf16 numbers, so they keep 16 significant bits.
//   window_attn_rows_kernel  fp32, and head sizes the others do not take: one CTA per (token, head), a warp per key.
#include "mdb_common.cuh"

namespace mdb {

// ---------------------------------------------------------------------------
// Queries, keys and values of a step
// ---------------------------------------------------------------------------
constexpr int kRotThreads = 256, kRotMaxPairs = 512;

// KEEP > 0: heads of up to 128 KEEP channels in registers, four per lane and step.
template <typename T, int KEEP, bool PARTS>
__global__ void __launch_bounds__(kRotThreads) rotary_commit_kernel(const mdb_rotary_commit_args a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float2 cs[kRotMaxPairs];          // (cos, sin) of the row's angles
  const int64_t row = blockIdx.x;
  const int pos = a.row_pos[row];
  if (pos < 0) return;
  for (int i = threadIdx.x; i < a.rot_dims / 2; i += kRotThreads) {
    // the angle and its distance from the nearest full turn in fp64: a product rounded to fp32 would be off by
    // pos * 2^-24
    const double turns = static_cast<double>(pos) * a.inv_freq[i] * 0.15915494309189535;
    float sn, c;
    sincospif(2.0f * static_cast<float>(turns - rint(turns)), &sn, &c);
    cs[i] = make_float2(c, sn);
  }
  __syncthreads();
  int64_t slot = a.slots[row];
  if (slot < -1 || slot >= a.num_slots) {
    if (threadIdx.x == 0) report_status(MDB_STATUS_BAD_SLOT);
    slot = -1;
  }
  const int lane = threadIdx.x & 31;
#pragma unroll 2
  for (int unit = threadIdx.x >> 5; unit < a.heads + 2 * a.kv_heads; unit += kRotThreads / 32) {
    const int kind = unit < a.heads ? 0 : (unit < a.heads + a.kv_heads ? 1 : 2);      // q, k or v
    const int head = unit - (kind == 0 ? 0 : (kind == 1 ? a.heads : a.heads + a.kv_heads));
    if (kind > 0 && slot < 0) continue;
    // by value: a reference picked at run time would be read through memory at every use
    mdb_rows src = a.q;
    if (kind == 1) src = a.k;
    if (kind == 2) src = a.v;
    T* out = kind == 0 ? static_cast<T*>(a.q_out) + (row * a.heads + head) * a.dim_pad
                       : static_cast<T*>(kind == 1 ? a.k_cache : a.v_cache) + (slot * a.kv_heads + head) * a.dim_pad;
    const float* w = kind == 0 ? a.q_norm : a.k_norm;
    if constexpr (KEEP > 0) {
      constexpr int kKeep = KEEP;
      float4 x[kKeep];
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < kKeep; ++i) {
        const int c = lane * 4 + 128 * i;
        x[i] = c < a.dim ? rows_at4_of<T, PARTS>(src, row, head * a.dim + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        ss += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
      }
      const float rstd = kind == 2 ? 1.0f : 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(a.dim) + a.eps);
#pragma unroll
      for (int i = 0; i < kKeep; ++i) {
        const int c = lane * 4 + 128 * i;
        if (c >= a.dim) continue;
        float4 y = x[i];
        if (kind < 2) {
          const float4 wv = *reinterpret_cast<const float4*>(w + c);
          y = make_float4(y.x * rstd * wv.x, y.y * rstd * wv.y, y.z * rstd * wv.z, y.w * rstd * wv.w);
          if (c < a.rot_dims) {
            const float2 r = cs[c / 2];
            y = make_float4(y.x * r.x - y.y * r.y, y.y * r.x + y.x * r.y, y.z, y.w);
          }
          if (c + 2 < a.rot_dims) {
            const float2 r = cs[c / 2 + 1];
            y = make_float4(y.x, y.y, y.z * r.x - y.w * r.y, y.w * r.x + y.z * r.y);
          }
        }
        act_store4(out + c, y);
      }
    } else {
      float ss = 0.f;
      for (int c = lane; c < a.dim; c += 32) {
        const float v = rows_at<T>(src, row, head * a.dim + c);
        ss += v * v;
      }
      const float rstd = 1.0f / sqrtf(warp_sum(ss) / static_cast<float>(a.dim) + a.eps);
      for (int c = lane; c < a.dim; c += 32) {
        const float v = rows_at<T>(src, row, head * a.dim + c);
        if (kind == 2) {
          out[c] = act_from_f<T>(v);
          continue;
        }
        float y = v * rstd * w[c];
        if (c < a.rot_dims) {                  // the pair's other channel (rot_dims is even)
          const float o = rows_at<T>(src, row, head * a.dim + (c ^ 1)) * rstd * w[c ^ 1];
          const float2 r = cs[c / 2];
          y = (c & 1) ? y * r.x + o * r.y : y * r.x - o * r.y;
        }
        out[c] = act_from_f<T>(y);
      }
    }
  }
}

// ---------------------------------------------------------------------------
// Attention of a few tokens
// ---------------------------------------------------------------------------
struct WinArgs {
  const void* q;              // [m][heads][dim_pad]
  const void* k_cache;        // [pages * 256][kv_heads][dim_pad]
  const void* v_cache;
  void* out;                  // [m] rows of ld_out, head h at column h * dim
  float* part_o;              // [m][nsplit][heads][dim_pad]
  float2* part_ml;            // [m][nsplit][heads]   (max in log2 units, sum)
  const int32_t* table;
  const int32_t* row_seq;
  const int32_t* row_pos;     // position of the row's token; -1: padding row
  int64_t ld_out;
  int table_stride, num_pages, m, heads, kv_heads, dim, dim_pad, window, sink, nsplit;
  float scale_log2, out_scale;
  mdb_rows gate;
};

__device__ __forceinline__ int win_page(const WinArgs& a, const int32_t* table, int index) {
  int page = index < a.table_stride ? table[index] : -1;
  if (page < 0 || page >= a.num_pages) {
    report_status(MDB_STATUS_BAD_PAGE);
    page = 0;
  }
  return page;
}
__device__ __forceinline__ int win_first(const WinArgs& a, int pos) { return a.window > 0 ? max(0, pos - a.window + 1) : 0; }

// factor of a head's weighted sum of values: output scale and gate over the softmax's denominator, whose sum l is in
// units of 2^m
template <typename T>
__device__ __forceinline__ float win_factor(const WinArgs& a, int64_t row, int head, float m, float l) {
  const float den = a.sink ? l + exp2f(-m) : l;
  const float g = rows_present(a.gate) ? sigmoid_f(rows_at<T>(a.gate, row, head)) : 1.0f;
  return a.out_scale * g / den;
}

constexpr int kWinKeys = 16, kWinHeads = 16, kWinWarps = 4, kWinStages = 3;

template <int DP>
struct WinPlan {
  static constexpr int kStride = DP + 8;                             // bf16 elements; the pad spreads rows over the banks
  static constexpr int kTile = kWinKeys * kStride * 2;               // bytes of a K or a V tile
  static constexpr int kRing = kWinStages * 2 * kTile;               // of one warp
  static constexpr int kMerge = kWinWarps * kWinHeads * (DP + 4) * 4 + kWinWarps * kWinHeads * 8;
  static constexpr int kBytes = kWinWarps * kRing > kMerge ? kWinWarps * kRing : kMerge;
};

// tiles of 16 keys (counted from the window's first one) that a key-range part covers: a multiple of the warps
__device__ __forceinline__ int win_part_tiles(int tiles, int nsplit) {
  return ((tiles + nsplit - 1) / nsplit + kWinWarps - 1) / kWinWarps * kWinWarps;
}

template <int DP>
__global__ void __launch_bounds__(kWinWarps * 32) window_attn_mma_kernel(const WinArgs a, const int head_blocks) {
  using P = WinPlan<DP>;
  constexpr int KS = DP / 16;              // k steps of the scores; column tiles of the output in pairs
  extern __shared__ __align__(16) unsigned char win_smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.z, split = blockIdx.x;
  const int kvh = blockIdx.y / head_blocks, block = blockIdx.y % head_blocks;
  const int group = a.heads / a.kv_heads;
  const int head0 = kvh * group + block * kWinHeads, nh = min(kWinHeads, group - block * kWinHeads);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = a.row_pos[row];
  if (pos < 0) return;
  const int lo = win_first(a, pos), hi = pos + 1, base_key = lo / kWinKeys * kWinKeys;
  const int tiles = (hi - base_key + kWinKeys - 1) / kWinKeys, part = win_part_tiles(tiles, a.nsplit);
  const int t_begin = split * part, t_end = min(tiles, t_begin + part);
  if (t_begin >= t_end) {                  // (never with one part)
    if (threadIdx.x < nh)
      a.part_ml[(static_cast<int64_t>(row) * a.nsplit + split) * a.heads + head0 + threadIdx.x] = make_float2(-INFINITY, 0.f);
    return;
  }
  const int32_t* table = a.table + static_cast<int64_t>(a.row_seq[row]) * a.table_stride;
  const uint32_t ring = smem_u32(win_smem) + warp * P::kRing;
  const int g = lane >> 2, j2 = 2 * (lane & 3);
  // q of the 16 heads as operand fragments (rows past the group: zeros)
  uint32_t qf[KS][4];
  {
    const bf16* q = static_cast<const bf16*>(a.q) + (static_cast<int64_t>(row) * a.heads + head0) * DP;
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int h = g + 8 * (i & 1), c = 16 * k + j2 + 8 * (i >> 1);
        qf[k][i] = h < nh ? *reinterpret_cast<const uint32_t*>(q + static_cast<int64_t>(h) * DP + c) : 0u;
      }
  }
  int page_index = -1, page = 0;
  auto load_tile = [&](int t, int stage) {
    if (t < t_end) {
      const int key0 = base_key + t * kWinKeys;
      if (key0 / kPage != page_index) {
        page_index = key0 / kPage;
        page = win_page(a, table, page_index);
      }
      const int64_t slot0 = static_cast<int64_t>(page) * kPage + key0 % kPage;
      const uint32_t dst = ring + stage * 2 * P::kTile;
#pragma unroll
      for (int i = 0; i < DP / 16; ++i) {
        const int idx = lane + 32 * i, key = idx / (DP / 8), c = idx % (DP / 8) * 8;
        const bool live = key0 + key >= lo && key0 + key < hi;
        const int64_t off = live ? ((slot0 + key) * a.kv_heads + kvh) * DP + c : 0;
        const uint32_t d = dst + (key * P::kStride + c) * 2;
        // a key outside the window: zeros (size 0 reads nothing), so that 0 * row stays 0
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(static_cast<const bf16*>(a.k_cache) + off),
                     "r"(live ? 16 : 0) : "memory");
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d + P::kTile), "l"(static_cast<const bf16*>(a.v_cache) + off),
                     "r"(live ? 16 : 0) : "memory");
      }
    }
    cp_async_commit();
  };
  const int t0 = t_begin + warp;
#pragma unroll
  for (int s = 0; s < kWinStages - 1; ++s) load_tile(t0 + s * kWinWarps, s);
  float acc[2 * KS][4];
#pragma unroll
  for (int i = 0; i < 2 * KS; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;      // of heads g and g + 8 (l: this lane's keys only)
  const uint32_t k_off = (((lane & 7) + ((lane >> 4) & 1) * 8) * P::kStride + ((lane >> 3) & 1) * 8) * 2;
  const uint32_t v_off = (((lane & 7) + ((lane >> 3) & 1) * 8) * P::kStride + (lane >> 4) * 8) * 2;
  int stage = 0;
  for (int t = t0; t < t_end; t += kWinWarps) {
    cp_async_wait<kWinStages - 2>();
    __syncwarp();                          // tile t has landed for the whole warp, tile t - 1 is consumed
    load_tile(t + (kWinStages - 1) * kWinWarps, stage == 0 ? kWinStages - 1 : stage - 1);
    const uint32_t kt = ring + stage * 2 * P::kTile, vt = kt + P::kTile;
    stage = stage + 1 == kWinStages ? 0 : stage + 1;
    float sc[2][2][4];                     // [parity of the k step][keys 0..7, 8..15]
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int n = 0; n < 2; ++n) sc[i][n][0] = sc[i][n][1] = sc[i][n][2] = sc[i][n][3] = 0.f;
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      uint32_t b[4];
      ldsm4(kt + k_off + 32 * k, b);
      mma16816(sc[k & 1][0], qf[k], b[0], b[1]);
      mma16816(sc[k & 1][1], qf[k], b[2], b[3]);
    }
    const int key = base_key + t * kWinKeys + j2;
    float x[2][4];                         // [keys 0..7, 8..15][head g: two keys, head g + 8: two keys]
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int kk = key + 8 * n + (e & 1);
        x[n][e] = kk >= lo && kk < hi ? (sc[0][n][e] + sc[1][n][e]) * a.scale_log2 : -INFINITY;
      }
    float mx0 = fmaxf(fmaxf(x[0][0], x[0][1]), fmaxf(x[1][0], x[1][1])), mx1 = fmaxf(fmaxf(x[0][2], x[0][3]), fmaxf(x[1][2], x[1][3]));
#pragma unroll
    for (int o = 1; o <= 2; o <<= 1) {
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, o));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, o));
    }
    // finite: every tile holds at least one key of the window
    const float n0 = fmaxf(m0, mx0), n1 = fmaxf(m1, mx1);
    if (__any_sync(0xffffffffu, n0 > m0 || n1 > m1)) {
      const float f0 = exp2f(m0 - n0), f1 = exp2f(m1 - n1);
      l0 *= f0;
      l1 *= f1;
#pragma unroll
      for (int i = 0; i < 2 * KS; ++i) { acc[i][0] *= f0; acc[i][1] *= f0; acc[i][2] *= f1; acc[i][3] *= f1; }
      m0 = n0;
      m1 = n1;
    }
    uint32_t ph[4], pl[4];
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const float p0 = exp2f(x[n][0] - m0), p1 = exp2f(x[n][1] - m0), p2 = exp2f(x[n][2] - m1), p3 = exp2f(x[n][3] - m1);
      l0 += p0 + p1;
      l1 += p2 + p3;
      const float h0 = bf16_round(p0), h1 = bf16_round(p1), h2 = bf16_round(p2), h3 = bf16_round(p3);
      ph[2 * n] = pack_bf16x2(h0, h1);
      ph[2 * n + 1] = pack_bf16x2(h2, h3);
      pl[2 * n] = pack_bf16x2(p0 - h0, p1 - h1);
      pl[2 * n + 1] = pack_bf16x2(p2 - h2, p3 - h3);
    }
#pragma unroll
    for (int i = 0; i < KS; ++i) {
      uint32_t v[4];                       // keys 0..15 of sixteen columns
      ldsm4_t(vt + v_off + 32 * i, v);
      mma16816(acc[2 * i], ph, v[0], v[1]);
      mma16816(acc[2 * i + 1], ph, v[2], v[3]);
      mma16816(acc[2 * i], pl, v[0], v[1]);
      mma16816(acc[2 * i + 1], pl, v[2], v[3]);
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int o = 1; o <= 2; o <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, o);
    l1 += __shfl_xor_sync(0xffffffffu, l1, o);
  }
  // the four warps' sums meet in shared memory
  constexpr int OS = DP + 4;
  float* so = reinterpret_cast<float*>(win_smem);                                    // [warps][16][OS]
  float2* sml = reinterpret_cast<float2*>(so + kWinWarps * kWinHeads * OS);          // [warps][16]
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2 * KS; ++i) {
    float* o = so + (warp * kWinHeads + g) * OS + 8 * i + j2;
    *reinterpret_cast<float2*>(o) = make_float2(acc[i][0], acc[i][1]);
    *reinterpret_cast<float2*>(o + 8 * OS) = make_float2(acc[i][2], acc[i][3]);
  }
  if ((lane & 3) == 0) {
    sml[warp * kWinHeads + g] = make_float2(m0, l0);
    sml[warp * kWinHeads + g + 8] = make_float2(m1, l1);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * (DP / 4); i += kWinWarps * 32) {
    const int h = i / (DP / 4), c = i % (DP / 4) * 4, head = head0 + h;
    float m = -INFINITY, l = 0.f;
#pragma unroll
    for (int w = 0; w < kWinWarps; ++w) m = fmaxf(m, sml[w * kWinHeads + h].x);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < kWinWarps; ++w) {
      const float2 ml = sml[w * kWinHeads + h];
      const float f = ml.x == -INFINITY ? 0.f : exp2f(ml.x - m);
      const float4 v = *reinterpret_cast<const float4*>(so + (w * kWinHeads + h) * OS + c);
      l = fmaf(f, ml.y, l);
      o.x = fmaf(f, v.x, o.x); o.y = fmaf(f, v.y, o.y); o.z = fmaf(f, v.z, o.z); o.w = fmaf(f, v.w, o.w);
    }
    if (a.nsplit == 1) {
      const float f = win_factor<bf16>(a, row, head, m, l);
      bf16* out = static_cast<bf16*>(a.out) + row * a.ld_out + static_cast<int64_t>(head) * a.dim + c;
      const float e[4] = {o.x * f, o.y * f, o.z * f, o.w * f};
#pragma unroll
      for (int k = 0; k < 4; ++k)
        if (c + k < a.dim) out[k] = __float2bfloat16_rn(e[k]);
    } else {
      const int64_t p = (static_cast<int64_t>(row) * a.nsplit + split) * a.heads + head;
      *reinterpret_cast<float4*>(a.part_o + p * DP + c) = o;
      if (c == 0) a.part_ml[p] = make_float2(m, l);
    }
  }
}

// One CTA per (head, row): the key-range parts weighted by their maxima.
__global__ void __launch_bounds__(64) window_combine_kernel(const WinArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.y, head = blockIdx.x;
  if (a.row_pos[row] < 0) return;
  const int64_t p0 = static_cast<int64_t>(row) * a.nsplit * a.heads + head;
  float m = -INFINITY, l = 0.f;
  for (int s = 0; s < a.nsplit; ++s) m = fmaxf(m, a.part_ml[p0 + static_cast<int64_t>(s) * a.heads].x);
  for (int s = 0; s < a.nsplit; ++s) {
    const float2 ml = a.part_ml[p0 + static_cast<int64_t>(s) * a.heads];
    l += ml.y * exp2f(ml.x - m);
  }
  const float f = win_factor<bf16>(a, row, head, m, l);
  bf16* out = static_cast<bf16*>(a.out) + row * a.ld_out + static_cast<int64_t>(head) * a.dim;
  for (int c = threadIdx.x * 4; c < a.dim; c += 256) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < a.nsplit; ++s) {
      const int64_t p = p0 + static_cast<int64_t>(s) * a.heads;
      const float pm = a.part_ml[p].x;
      if (pm == -INFINITY) continue;       // an empty part left its accumulator unwritten
      const float w = exp2f(pm - m) * f;
      const float4 v = *reinterpret_cast<const float4*>(a.part_o + p * a.dim_pad + c);
      o.x = fmaf(w, v.x, o.x); o.y = fmaf(w, v.y, o.y); o.z = fmaf(w, v.z, o.z); o.w = fmaf(w, v.w, o.w);
    }
    const float e[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (c + k < a.dim) out[c + k] = __float2bfloat16_rn(e[k]);
  }
}

// One CTA of four warps per (head, row); warp w takes keys first + w, + 4, ...; a lane owns every 32nd group of four
// channels.  NV = channels per lane / 4.
template <typename T, int NV>
__global__ void __launch_bounds__(128) window_attn_rows_kernel(const WinArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sm[4], sl[4];
  extern __shared__ float win_rows_o[];        // [4][dim_pad]
  const int row = blockIdx.y, head = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = a.row_pos[row];
  if (pos < 0) return;
  const int kvh = head / (a.heads / a.kv_heads);
  const int32_t* table = a.table + static_cast<int64_t>(a.row_seq[row]) * a.table_stride;
  const T* q = static_cast<const T*>(a.q) + (static_cast<int64_t>(row) * a.heads + head) * a.dim_pad;
  float4 qv[NV], o[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    qv[i] = o[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    const int c = (lane + 32 * i) * 4;
    if (c < a.dim_pad) qv[i] = act_load4(q + c);
  }
  float m = -INFINITY, l = 0.f;
  for (int key = win_first(a, pos) + warp; key <= pos; key += 4) {
    const int64_t slot = static_cast<int64_t>(win_page(a, table, key / kPage)) * kPage + key % kPage;
    const int64_t off = (slot * a.kv_heads + kvh) * a.dim_pad;
    const T* kr = static_cast<const T*>(a.k_cache) + off;
    const T* vr = static_cast<const T*>(a.v_cache) + off;
    float4 vv[NV];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      float4 kv = make_float4(0.f, 0.f, 0.f, 0.f);
      vv[i] = kv;
      const int c = (lane + 32 * i) * 4;
      if (c < a.dim_pad) {
        kv = act_load4(kr + c);
        vv[i] = act_load4(vr + c);
      }
      s += qv[i].x * kv.x + qv[i].y * kv.y + qv[i].z * kv.z + qv[i].w * kv.w;
    }
    s = warp_sum(s) * a.scale_log2;
    const float m_new = fmaxf(m, s), f = exp2f(m - m_new), p = exp2f(s - m_new);
    m = m_new;
    l = l * f + p;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      o[i].x = fmaf(p, vv[i].x, o[i].x * f); o[i].y = fmaf(p, vv[i].y, o[i].y * f);
      o[i].z = fmaf(p, vv[i].z, o[i].z * f); o[i].w = fmaf(p, vv[i].w, o[i].w * f);
    }
  }
  if (lane == 0) { sm[warp] = m; sl[warp] = l; }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (lane + 32 * i) * 4;
    if (c < a.dim_pad) *reinterpret_cast<float4*>(win_rows_o + warp * a.dim_pad + c) = o[i];
  }
  __syncthreads();
  const float mx = fmaxf(fmaxf(sm[0], sm[1]), fmaxf(sm[2], sm[3]));
  float w[4], total = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    w[i] = sm[i] == -INFINITY ? 0.f : exp2f(sm[i] - mx);
    total += w[i] * sl[i];
  }
  const float f = win_factor<T>(a, row, head, mx, total);
  T* out = static_cast<T*>(a.out) + row * a.ld_out + static_cast<int64_t>(head) * a.dim;
  for (int c = threadIdx.x; c < a.dim; c += 128)
    out[c] = act_from_f<T>((w[0] * win_rows_o[c] + w[1] * win_rows_o[a.dim_pad + c] + w[2] * win_rows_o[2 * a.dim_pad + c] +
                            w[3] * win_rows_o[3 * a.dim_pad + c]) * f);
}

template <int DP>
static int launch_window_mma(const WinArgs& a, cudaStream_t st) {
  static PerDeviceOnce attr_once;
  const int dev = attr_once.slot();
  if (dev < 0) return MDB_ERR_CUDA;
  if (!attr_once.done[dev]) {
    if (cudaFuncSetAttribute(window_attn_mma_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, WinPlan<DP>::kBytes) != cudaSuccess)
      return MDB_ERR_CUDA;
    attr_once.done[dev] = true;
  }
  const int head_blocks = (a.heads / a.kv_heads + kWinHeads - 1) / kWinHeads;
  if (a.kv_heads * head_blocks > 65535) return MDB_ERR_UNSUPPORTED;
  int rc = mdb_launch(window_attn_mma_kernel<DP>, dim3(a.nsplit, a.kv_heads * head_blocks, a.m), dim3(kWinWarps * 32), WinPlan<DP>::kBytes, st, a,
                      head_blocks);
  if (rc == MDB_OK && a.nsplit > 1) rc = mdb_launch(window_combine_kernel, dim3(a.heads, a.m), dim3(64), 0, st, a);
  return rc;
}

template <typename T>
static int launch_window_rows(const WinArgs& a, cudaStream_t st) {
  const dim3 grid(a.heads, a.m);
  const size_t smem = 4 * sizeof(float) * a.dim_pad;
  if (a.dim_pad <= 128) return mdb_launch(window_attn_rows_kernel<T, 1>, grid, dim3(128), smem, st, a);
  if (a.dim_pad <= 256) return mdb_launch(window_attn_rows_kernel<T, 2>, grid, dim3(128), smem, st, a);
  if (a.dim_pad <= 512) return mdb_launch(window_attn_rows_kernel<T, 4>, grid, dim3(128), smem, st, a);
  if (a.dim_pad <= 1024) return mdb_launch(window_attn_rows_kernel<T, 8>, grid, dim3(128), smem, st, a);
  return MDB_ERR_UNSUPPORTED;
}

// longest portion that still goes token by token
constexpr int kWinRowsMaxPortion = 8;

}  // namespace mdb

using namespace mdb;

extern "C" {

int mdb_rotary_commit(const mdb_rotary_commit_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_rotary_commit_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.heads > 0 && a.kv_heads > 0 && a.dim > 0 && a.dim_pad >= a.dim, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(a.rot_dims >= 0 && a.rot_dims <= a.dim && a.rot_dims % 2 == 0, MDB_ERR_ARG);
  MDB_REQUIRE(rows_present(a.q) && rows_present(a.k) && rows_present(a.v) && a.q_norm && a.k_norm && (a.inv_freq || a.rot_dims == 0) &&
                  a.row_pos && a.slots && a.q_out && a.k_cache && a.v_cache,
              MDB_ERR_ARG);
  MDB_REQUIRE(a.rot_dims / 2 <= kRotMaxPairs, MDB_ERR_UNSUPPORTED);
  const bool parts = a.q.parts != nullptr;
  MDB_REQUIRE((a.k.parts != nullptr) == parts && (a.v.parts != nullptr) == parts && (!parts || a.dtype == MDB_BF16), MDB_ERR_UNSUPPORTED);
  const bool vec = a.dim % 4 == 0 && a.dim <= 256 && a.dim_pad % 4 == 0 && rows_ok(a.q) && rows_ok(a.k) && rows_ok(a.v) &&
                   mdb_aligned16(a.q_norm) && mdb_aligned16(a.k_norm) && mdb_aligned16(a.q_out) && mdb_aligned16(a.k_cache) && mdb_aligned16(a.v_cache);
  const dim3 grid(a.m), block(kRotThreads);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a.dtype == MDB_F32)
    return vec ? mdb_launch(rotary_commit_kernel<float, 2, false>, grid, block, 0, st, a)
               : mdb_launch(rotary_commit_kernel<float, 0, false>, grid, block, 0, st, a);
  if (!vec) return mdb_launch(rotary_commit_kernel<bf16, 0, false>, grid, block, 0, st, a);
  if (parts)
    return a.dim <= 128 ? mdb_launch(rotary_commit_kernel<bf16, 1, true>, grid, block, 0, st, a)
                        : mdb_launch(rotary_commit_kernel<bf16, 2, true>, grid, block, 0, st, a);
  return a.dim <= 128 ? mdb_launch(rotary_commit_kernel<bf16, 1, false>, grid, block, 0, st, a)
                      : mdb_launch(rotary_commit_kernel<bf16, 2, false>, grid, block, 0, st, a);
}

int64_t mdb_window_attn_workspace_bytes(int m, int heads, int dim_pad, int nsplit) {
  if (m <= 0 || heads <= 0 || dim_pad <= 0 || nsplit <= 1) return 0;
  return static_cast<int64_t>(m) * nsplit * heads * (dim_pad + 2) * 4;
}

int mdb_window_attn(const mdb_window_attn_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_window_attn_args w = *args;
  MDB_REQUIRE(w.m >= 0 && w.bs >= 0 && w.heads > 0 && w.kv_heads > 0 && w.heads % w.kv_heads == 0 && w.dim > 0 && w.dim_pad >= w.dim &&
                  w.window >= 0 && w.num_pages > 0 && w.table_stride > 0 && w.nsplit >= 1,
              MDB_ERR_ARG);
  if (w.m == 0) return MDB_OK;
  MDB_REQUIRE(w.q && w.k_cache && w.v_cache && w.out && w.block_table && w.row_seq && w.row_pos, MDB_ERR_ARG);
  MDB_REQUIRE(w.ld_out >= static_cast<int64_t>(w.heads) * w.dim, MDB_ERR_ARG);
  MDB_REQUIRE(w.dim_pad % 8 == 0 && w.ld_out % 8 == 0 && mdb_aligned16(w.q) && mdb_aligned16(w.k_cache) && mdb_aligned16(w.v_cache) &&
                  mdb_aligned16(w.out) && mdb_aligned16(w.workspace),
              MDB_ERR_ALIGN);
  MDB_REQUIRE(w.m <= 65535 && w.heads <= 65535, MDB_ERR_UNSUPPORTED);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (w.max_q > kWinRowsMaxPortion && attn_win_tc_supported(w)) return attn_win_tc_launch(w, st);
  WinArgs a = {};
  a.q = w.q; a.k_cache = w.k_cache; a.v_cache = w.v_cache; a.out = w.out;
  a.table = w.block_table; a.row_seq = w.row_seq; a.row_pos = w.row_pos;
  a.ld_out = w.ld_out;
  a.table_stride = w.table_stride; a.num_pages = w.num_pages;
  a.m = w.m; a.heads = w.heads; a.kv_heads = w.kv_heads; a.dim = w.dim; a.dim_pad = w.dim_pad;
  a.window = w.window; a.sink = w.sink;
  a.scale_log2 = w.scale * 1.4426950408889634f;
  a.out_scale = w.out_scale;
  a.gate = w.gate;
  a.nsplit = 1;
  if (w.dtype == MDB_F32) return launch_window_rows<float>(a, st);
  if (w.dim_pad != 64 && w.dim_pad != 128 && w.dim_pad != 192 && w.dim_pad != 256) return launch_window_rows<bf16>(a, st);
  a.nsplit = w.nsplit;
  const int64_t need = mdb_window_attn_workspace_bytes(w.m, w.heads, w.dim_pad, w.nsplit);
  MDB_REQUIRE(need == 0 || (w.workspace != nullptr && w.workspace_bytes >= need), MDB_ERR_WORKSPACE);
  a.part_o = static_cast<float*>(w.workspace);
  a.part_ml = a.part_o ? reinterpret_cast<float2*>(a.part_o + static_cast<int64_t>(w.m) * w.nsplit * w.heads * w.dim_pad) : nullptr;
  switch (w.dim_pad) {
    case 64: return launch_window_mma<64>(a, st);
    case 128: return launch_window_mma<128>(a, st);
    case 192: return launch_window_mma<192>(a, st);
    default: return launch_window_mma<256>(a, st);
  }
}

}  // extern "C"
