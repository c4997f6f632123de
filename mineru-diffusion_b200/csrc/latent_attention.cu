// Causal attention over cached latents: every query head of a token reads the same latent row of a key, which stands
// for its key and its value alike (the per-head key projection is folded into the query, the per-head value
// projection follows the attention), so a key costs one latent row of memory traffic for all heads.
//
//   latent_attn_mma_kernel   bf16: a CTA takes 16 heads of one token and a range of its keys (split over CTAs, merged by
//                            latent_combine_kernel).  Latent tiles of 32 keys come through a cp.async ring;
//                            scores and outputs are m16n8k16 products, the 16 heads being the 16 rows: a 128-row
//                            tile of the tensor-memory kind would be seven-eighths empty.  Softmax in fp32; the weights
//                            enter the second product as the sum of two bf16 numbers, so they keep 16 significant bits.
//   latent_attn_rows_kernel  fp32, and widths the first kernel does not take: one CTA per (token, head), a warp per key.
#include "mdb_common.cuh"

namespace mdb {

struct LatentArgs {
  const void* q;              // [m][heads][width]
  const void* cache;          // [pages * 256][width]
  void* out;                  // [m][heads][width]
  float* part_o;              // [m][nsplit][heads][width]
  float2* part_ml;            // [m][nsplit][heads]   (max in log2 units, sum)
  const int32_t* table;
  const int32_t* row_seq;
  const int32_t* row_pos;     // position of the row's token; -1: padding row
  int table_stride, num_pages, m, heads, width, nsplit;
  float scale_log2;
};

__device__ __forceinline__ int64_t latent_slot(const LatentArgs& a, const int32_t* table, int pos) {
  int page = pos / kPage < a.table_stride ? table[pos / kPage] : -1;
  if (page < 0 || page >= a.num_pages) {
    report_status(MDB_STATUS_BAD_PAGE);
    page = 0;
  }
  return static_cast<int64_t>(page) * kPage + pos % kPage;
}

// keys of one part of a context of n keys: a multiple of 32
__device__ __forceinline__ int latent_part(int n, int nsplit) { return ((n + nsplit - 1) / nsplit + 31) / 32 * 32; }

__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

constexpr int kLatKeys = 32, kLatHeads = 16, kLatThreads = 256;
constexpr int kLatPStride = kLatKeys + 8;
constexpr int kLatSStride = kLatKeys + 8;

template <int WIDTH>
struct LatPlan {
  static constexpr int kStride = WIDTH + 8;                    // bf16 elements; the pad spreads rows over the banks
  static constexpr int kTile = kLatKeys * kStride * 2;
  static constexpr int kStages = WIDTH > 256 ? 2 : 3;          // two CTAs per SM at every width
  static constexpr int kOffTiles = 0;
  static constexpr int kOffS = kOffTiles + kStages * kTile;                        // [8 warps][16][40] fp32 partial scores;
  static constexpr int kQBytes = kLatHeads * kStride * 2;                          // q passes through it on its way to registers
  static constexpr int kSBytes = 8 * kLatHeads * kLatSStride * 4;
  static constexpr int kOffP = kOffS + (kQBytes > kSBytes ? kQBytes : kSBytes);    // [2][16][40] bf16: high and low parts
  static constexpr int kOffF = kOffP + 2 * kLatHeads * kLatPStride * 2;            // [16] fp32
  static constexpr int kBytes = kOffF + 64;
};

template <int WIDTH>
__global__ void __launch_bounds__(kLatThreads) latent_attn_mma_kernel(const LatentArgs a) {
  using P = LatPlan<WIDTH>;
  constexpr int NT = WIDTH / 64;           // 8-column tiles of the output per warp
  extern __shared__ __align__(16) unsigned char lat_smem[];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.z, head0 = blockIdx.y * kLatHeads, split = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = a.row_pos[row];
  if (pos < 0) return;
  const int n = pos + 1, part = latent_part(n, a.nsplit);
  const int k_begin = split * part, k_end = min(n, k_begin + part);
  const int32_t* table = a.table + static_cast<int64_t>(a.row_seq[row]) * a.table_stride;
  const bf16* cache = static_cast<const bf16*>(a.cache);
  const int nh = min(kLatHeads, a.heads - head0);
  if (k_begin >= k_end) {
    if (a.nsplit > 1 && threadIdx.x < nh)
      a.part_ml[(static_cast<int64_t>(row) * a.nsplit + split) * a.heads + head0 + threadIdx.x] = make_float2(-INFINITY, 0.f);
    return;
  }
  const uint32_t base = smem_u32(lat_smem);
  bf16* qs = reinterpret_cast<bf16*>(lat_smem + P::kOffS);
  {
    const bf16* q = static_cast<const bf16*>(a.q) + (static_cast<int64_t>(row) * a.heads + head0) * WIDTH;
    for (int i = threadIdx.x; i < kLatHeads * (WIDTH / 8); i += kLatThreads) {
      const int h = i / (WIDTH / 8), c = i % (WIDTH / 8);
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (h < nh) v = *reinterpret_cast<const uint4*>(q + static_cast<int64_t>(h) * WIDTH + c * 8);
      *reinterpret_cast<uint4*>(qs + h * P::kStride + c * 8) = v;
    }
  }
  const int tiles = (k_end - k_begin + kLatKeys - 1) / kLatKeys;
  auto load_tile = [&](int t) {
    if (t < tiles) {
      const uint32_t dst = base + P::kOffTiles + (t % P::kStages) * P::kTile;
      const int key = threadIdx.x >> 3, pos_k = k_begin + t * kLatKeys + key;
      const bool live = pos_k < k_end;
      const bf16* src = cache + (live ? latent_slot(a, table, pos_k) : 0) * WIDTH;
#pragma unroll
      for (int i = 0; i < WIDTH / 64; ++i) {
        const int c = (threadIdx.x & 7) + 8 * i;
        // a key past the end of the part: zeros (size 0 reads nothing), so that 0 * row stays 0
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + (key * P::kStride + c * 8) * 2),
                     "l"(src + c * 8), "r"(live ? 16 : 0) : "memory");
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int t = 0; t < P::kStages - 1; ++t) load_tile(t);
  // warp w owns columns [w, w + 1) * WIDTH / 8 of q (in registers), of the scores' sum and of the output
  constexpr int KS = WIDTH / 128;          // k steps of 16 of a warp's share
  const int c_first = warp * (WIDTH / 8);
  uint32_t qf[KS][4];
  __syncthreads();
#pragma unroll
  for (int k = 0; k < KS; ++k) ldsm4(base + P::kOffS + ((lane & 15) * P::kStride + c_first + 16 * k + (lane >> 4) * 8) * 2, qf[k]);
  __syncthreads();                         // the scores' buffer is free
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  float* ss = reinterpret_cast<float*>(lat_smem + P::kOffS);
  bf16* ps = reinterpret_cast<bf16*>(lat_smem + P::kOffP);
  float* fs = reinterpret_cast<float*>(lat_smem + P::kOffF);
  const int srow = threadIdx.x >> 4, sj = threadIdx.x & 15;      // softmax: 16 threads per head, two keys each
  float m_run = -INFINITY, l_run = 0.f;                          // (l: this thread's keys only)
  const int g = lane >> 2;
  for (int t = 0; t < tiles; ++t) {
    cp_async_wait<P::kStages - 2>();
    __syncthreads();                       // tile t has landed, tile t - 1 is consumed
    load_tile(t + P::kStages - 1);
    const uint32_t tile = base + P::kOffTiles + (t % P::kStages) * P::kTile;
    {
      // scores of all 32 keys over this warp's columns: four independent products
      float sc[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        uint32_t b0[4], b1[4];             // first and second eight columns of the step, keys 0..31
        const uint32_t ka = tile + (lane * P::kStride + c_first + 16 * k) * 2;
        ldsm4(ka, b0);
        ldsm4(ka + 16, b1);
#pragma unroll
        for (int n = 0; n < 4; ++n) mma16816(sc[n], qf[k], b0[n], b1[n]);
      }
      float* so = ss + (warp * kLatHeads + g) * kLatSStride + 2 * (lane & 3);
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        *reinterpret_cast<float2*>(so + 8 * n) = make_float2(sc[n][0], sc[n][1]);
        *reinterpret_cast<float2*>(so + 8 * kLatSStride + 8 * n) = make_float2(sc[n][2], sc[n][3]);
      }
    }
    __syncthreads();
    {
      float2 sv[8];
#pragma unroll
      for (int w = 0; w < 8; ++w) sv[w] = *reinterpret_cast<const float2*>(ss + (w * kLatHeads + srow) * kLatSStride + 2 * sj);
      const float x0 = ((sv[0].x + sv[1].x) + (sv[2].x + sv[3].x)) + ((sv[4].x + sv[5].x) + (sv[6].x + sv[7].x));
      const float x1 = ((sv[0].y + sv[1].y) + (sv[2].y + sv[3].y)) + ((sv[4].y + sv[5].y) + (sv[6].y + sv[7].y));
      const int key = k_begin + t * kLatKeys + 2 * sj;
      const float a0 = key < k_end ? x0 * a.scale_log2 : -INFINITY;
      const float a1 = key + 1 < k_end ? x1 * a.scale_log2 : -INFINITY;
      float mx = fmaxf(a0, a1);
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_new = fmaxf(m_run, mx);         // finite: a tile holds at least one key
      const float f = exp2f(m_run - m_new), p0 = exp2f(a0 - m_new), p1 = exp2f(a1 - m_new);
      l_run = l_run * f + p0 + p1;
      m_run = m_new;
      const float h0 = bf16_round(p0), h1 = bf16_round(p1);
      *reinterpret_cast<uint32_t*>(ps + srow * kLatPStride + 2 * sj) = pack_bf16x2(h0, h1);
      *reinterpret_cast<uint32_t*>(ps + (kLatHeads + srow) * kLatPStride + 2 * sj) = pack_bf16x2(p0 - h0, p1 - h1);
      if (sj == 0) fs[srow] = f;
    }
    __syncthreads();
    {
      const float f0 = fs[g], f1 = fs[g + 8];
#pragma unroll
      for (int i = 0; i < NT; ++i) { acc[i][0] *= f0; acc[i][1] *= f0; acc[i][2] *= f1; acc[i][3] *= f1; }
      uint32_t ph[2][4], pl[2][4];
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        const uint32_t pa = base + P::kOffP + ((lane & 15) * kLatPStride + ks * 16 + (lane >> 4) * 8) * 2;
        ldsm4(pa, ph[ks]);
        ldsm4(pa + kLatHeads * kLatPStride * 2, pl[ks]);
      }
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        uint32_t v[4];                     // keys 0..31 of eight columns
        ldsm4_t(tile + (lane * P::kStride + c_first + 8 * i) * 2, v);
        mma16816(acc[i], ph[0], v[0], v[1]);
        mma16816(acc[i], pl[0], v[0], v[1]);
        mma16816(acc[i], ph[1], v[2], v[3]);
        mma16816(acc[i], pl[1], v[2], v[3]);
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int o = 8; o > 0; o >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, o);
  __syncthreads();
  if (sj == 0) fs[srow] = 1.0f / l_run;
  __syncthreads();
  const int c0 = c_first + 2 * (lane & 3);
  if (a.nsplit == 1) {
    bf16* out = static_cast<bf16*>(a.out) + (static_cast<int64_t>(row) * a.heads + head0) * WIDTH;
    const float f0 = fs[g], f1 = fs[g + 8];
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      if (g < nh) *reinterpret_cast<uint32_t*>(out + static_cast<int64_t>(g) * WIDTH + c0 + 8 * i) = pack_bf16x2(acc[i][0] * f0, acc[i][1] * f0);
      if (g + 8 < nh)
        *reinterpret_cast<uint32_t*>(out + static_cast<int64_t>(g + 8) * WIDTH + c0 + 8 * i) = pack_bf16x2(acc[i][2] * f1, acc[i][3] * f1);
    }
  } else {
    const int64_t p0 = (static_cast<int64_t>(row) * a.nsplit + split) * a.heads + head0;
    float* out = a.part_o + p0 * WIDTH;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      if (g < nh) *reinterpret_cast<float2*>(out + static_cast<int64_t>(g) * WIDTH + c0 + 8 * i) = make_float2(acc[i][0], acc[i][1]);
      if (g + 8 < nh) *reinterpret_cast<float2*>(out + static_cast<int64_t>(g + 8) * WIDTH + c0 + 8 * i) = make_float2(acc[i][2], acc[i][3]);
    }
    if (sj == 0 && srow < nh) a.part_ml[p0 + srow] = make_float2(m_run, l_run);
  }
}

// One CTA per (head, row): the key-range parts of a context weighted by their maxima.
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.y, head = blockIdx.x;
  if (a.row_pos[row] < 0) return;
  const int64_t p0 = static_cast<int64_t>(row) * a.nsplit * a.heads + head;
  float mx = -INFINITY;
  for (int s = 0; s < a.nsplit; ++s) mx = fmaxf(mx, a.part_ml[p0 + static_cast<int64_t>(s) * a.heads].x);
  float l = 0.f;
  for (int s = 0; s < a.nsplit; ++s) {
    const float2 ml = a.part_ml[p0 + static_cast<int64_t>(s) * a.heads];
    l += ml.y * exp2f(ml.x - mx);
  }
  const float inv = 1.0f / l;
  bf16* out = static_cast<bf16*>(a.out) + (static_cast<int64_t>(row) * a.heads + head) * a.width;
  for (int c = threadIdx.x * 4; c < a.width; c += 512) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < a.nsplit; ++s) {
      const int64_t p = p0 + static_cast<int64_t>(s) * a.heads;
      const float m = a.part_ml[p].x;
      if (m == -INFINITY) continue;        // an empty part left its accumulator unwritten
      const float w = exp2f(m - mx) * inv;
      const float4 v = *reinterpret_cast<const float4*>(a.part_o + p * a.width + c);
      o.x = fmaf(w, v.x, o.x); o.y = fmaf(w, v.y, o.y); o.z = fmaf(w, v.z, o.z); o.w = fmaf(w, v.w, o.w);
    }
    act_store4(out + c, o);
  }
}

// One CTA of four warps per (head, row); warp w takes keys w, w + 4, ...; a lane owns every 32nd float4 group of four
// channels.  NV = channels per lane / 4.
template <typename T, int NV>
__global__ void __launch_bounds__(128) latent_attn_rows_kernel(const LatentArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sm[4], sl[4];
  extern __shared__ float rows_o[];        // [4][width]
  const int row = blockIdx.y, head = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = a.row_pos[row];
  if (pos < 0) return;
  const int32_t* table = a.table + static_cast<int64_t>(a.row_seq[row]) * a.table_stride;
  const T* q = static_cast<const T*>(a.q) + (static_cast<int64_t>(row) * a.heads + head) * a.width;
  float4 qv[NV], o[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    qv[i] = o[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    const int c = (lane + 32 * i) * 4;
    if (c < a.width) qv[i] = act_load4(q + c);
  }
  float m = -INFINITY, l = 0.f;
  for (int key = warp; key <= pos; key += 4) {
    const T* kr = static_cast<const T*>(a.cache) + latent_slot(a, table, key) * a.width;
    float4 kv[NV];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      kv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      const int c = (lane + 32 * i) * 4;
      if (c < a.width) kv[i] = act_load4(kr + c);
      s += qv[i].x * kv[i].x + qv[i].y * kv[i].y + qv[i].z * kv[i].z + qv[i].w * kv[i].w;
    }
    s = warp_sum(s) * a.scale_log2;
    const float m_new = fmaxf(m, s), f = exp2f(m - m_new), p = exp2f(s - m_new);
    m = m_new;
    l = l * f + p;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      o[i].x = fmaf(p, kv[i].x, o[i].x * f); o[i].y = fmaf(p, kv[i].y, o[i].y * f);
      o[i].z = fmaf(p, kv[i].z, o[i].z * f); o[i].w = fmaf(p, kv[i].w, o[i].w * f);
    }
  }
  if (lane == 0) { sm[warp] = m; sl[warp] = l; }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (lane + 32 * i) * 4;
    if (c < a.width) *reinterpret_cast<float4*>(rows_o + warp * a.width + c) = o[i];
  }
  __syncthreads();
  const float mx = fmaxf(fmaxf(sm[0], sm[1]), fmaxf(sm[2], sm[3]));
  float w[4], total = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    w[i] = sm[i] == -INFINITY ? 0.f : exp2f(sm[i] - mx);
    total += w[i] * sl[i];
  }
  T* out = static_cast<T*>(a.out) + (static_cast<int64_t>(row) * a.heads + head) * a.width;
  for (int c = threadIdx.x; c < a.width; c += 128)
    out[c] = act_from_f<T>((w[0] * rows_o[c] + w[1] * rows_o[a.width + c] + w[2] * rows_o[2 * a.width + c] + w[3] * rows_o[3 * a.width + c]) / total);
}

template <int WIDTH>
static int launch_latent_mma(const LatentArgs& a, cudaStream_t st) {
  static PerDeviceOnce attr_once;
  const int dev = attr_once.slot();
  if (dev < 0) return MDB_ERR_CUDA;
  if (!attr_once.done[dev]) {
    if (cudaFuncSetAttribute(latent_attn_mma_kernel<WIDTH>, cudaFuncAttributeMaxDynamicSharedMemorySize, LatPlan<WIDTH>::kBytes) != cudaSuccess)
      return MDB_ERR_CUDA;
    attr_once.done[dev] = true;
  }
  const dim3 grid(a.nsplit, (a.heads + kLatHeads - 1) / kLatHeads, a.m);
  int rc = mdb_launch(latent_attn_mma_kernel<WIDTH>, grid, dim3(kLatThreads), LatPlan<WIDTH>::kBytes, st, a);
  if (rc == MDB_OK && a.nsplit > 1) rc = mdb_launch(latent_combine_kernel, dim3(a.heads, a.m), dim3(128), 0, st, a);
  return rc;
}

template <typename T>
static int launch_latent_rows(const LatentArgs& a, cudaStream_t st) {
  const dim3 grid(a.heads, a.m);
  const size_t smem = 4 * sizeof(float) * a.width;
  if (a.width <= 128) return mdb_launch(latent_attn_rows_kernel<T, 1>, grid, dim3(128), smem, st, a);
  if (a.width <= 256) return mdb_launch(latent_attn_rows_kernel<T, 2>, grid, dim3(128), smem, st, a);
  if (a.width <= 512) return mdb_launch(latent_attn_rows_kernel<T, 4>, grid, dim3(128), smem, st, a);
  if (a.width <= 1024) return mdb_launch(latent_attn_rows_kernel<T, 8>, grid, dim3(128), smem, st, a);
  if (a.width <= 2048) return mdb_launch(latent_attn_rows_kernel<T, 16>, grid, dim3(128), smem, st, a);
  return MDB_ERR_UNSUPPORTED;
}

static bool latent_mma_width(int width) { return width == 128 || width == 256 || width == 384 || width == 512; }

}  // namespace mdb

using namespace mdb;

extern "C" {

int64_t mdb_latent_attn_workspace_bytes(int m, int heads, int width, int nsplit) {
  if (m <= 0 || heads <= 0 || width <= 0 || nsplit <= 1) return 0;
  return static_cast<int64_t>(m) * nsplit * heads * (width + 2) * 4;
}

int mdb_latent_attn(int dtype, const void* q, const void* cache, void* out, const int32_t* block_table, int table_stride,
                    const int32_t* row_seq, const int32_t* row_pos, int m, int heads, int width, int num_pages, float scale,
                    int nsplit, void* workspace, int64_t workspace_bytes, mdb_stream_t stream) {
  MDB_REQUIRE(m >= 0 && heads > 0 && width > 0 && num_pages > 0 && table_stride > 0 && nsplit >= 1, MDB_ERR_ARG);
  if (m == 0) return MDB_OK;
  MDB_REQUIRE(q && cache && out && block_table && row_seq && row_pos, MDB_ERR_ARG);
  MDB_REQUIRE(width % 8 == 0 && mdb_aligned16(q) && mdb_aligned16(cache) && mdb_aligned16(out) && mdb_aligned16(workspace), MDB_ERR_ALIGN);
  MDB_REQUIRE(m <= 65535, MDB_ERR_UNSUPPORTED);
  LatentArgs a = {};
  a.q = q; a.cache = cache; a.out = out;
  a.table = block_table; a.table_stride = table_stride; a.num_pages = num_pages;
  a.row_seq = row_seq; a.row_pos = row_pos;
  a.m = m; a.heads = heads; a.width = width;
  a.scale_log2 = scale * 1.4426950408889634f;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == MDB_F32 || !latent_mma_width(width)) {
    a.nsplit = 1;
    return dtype == MDB_F32 ? launch_latent_rows<float>(a, st) : launch_latent_rows<bf16>(a, st);
  }
  a.nsplit = nsplit;
  const int64_t need = mdb_latent_attn_workspace_bytes(m, heads, width, nsplit);
  MDB_REQUIRE(need == 0 || (workspace != nullptr && workspace_bytes >= need), MDB_ERR_WORKSPACE);
  a.part_o = static_cast<float*>(workspace);
  a.part_ml = a.part_o ? reinterpret_cast<float2*>(a.part_o + static_cast<int64_t>(m) * nsplit * heads * width) : nullptr;
  switch (width) {
    case 128: return launch_latent_mma<128>(a, st);
    case 256: return launch_latent_mma<256>(a, st);
    case 384: return launch_latent_mma<384>(a, st);
    default: return launch_latent_mma<512>(a, st);
  }
}

}  // extern "C"
