// Mixture of experts: group-limited top-k routing, the plan that lays the chosen (token, expert) pairs out by expert
// in tiles of 128 rows (the unit of the grouped GEMMs), and the row gather into that layout.
#include "mdb_common.cuh"

namespace mdb {

constexpr int kMoeTileRows = 128;      // rows of one expert start on a multiple of this
constexpr int kRouteWarps = 4;

// One warp per token.  Scores = softmax of the fp32 router logits over all experts; a group's score is its largest;
// the best `keep` groups stay in play; the `top` largest remaining scores win (ties to the lower index), and their
// weights are the scores divided by (their sum + 1e-20).
__global__ void __launch_bounds__(kRouteWarps * 32) moe_route_kernel(const mdb_moe_route_args a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float route_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t row = static_cast<int64_t>(blockIdx.x) * kRouteWarps + warp;
  if (row >= a.m) return;
  float* s = route_smem + warp * (a.experts + a.groups);
  float* gs = s + a.experts;
  if (a.row_slot != nullptr && a.row_slot[row] < 0) {       // padding row of a batch: routed nowhere
    for (int k = lane; k < a.top; k += 32) a.ids[row * a.top + k] = -1;
    return;
  }
  float mx = -INFINITY;
  for (int e = lane; e < a.experts; e += 32) {
    const float z = rows_at<float>(a.logits, row, e);
    s[e] = z;
    mx = fmaxf(mx, z);
  }
  mx = warp_max(mx);
  float sum = 0.f;
  for (int e = lane; e < a.experts; e += 32) {
    const float p = expf(s[e] - mx);
    s[e] = p;
    sum += p;
  }
  sum = warp_sum(sum);
  const float inv = 1.0f / sum;
  for (int e = lane; e < a.experts; e += 32) s[e] *= inv;
  __syncwarp();
  if (a.groups > 1 && a.keep < a.groups) {
    const int size = a.experts / a.groups;
    for (int g = lane; g < a.groups; g += 32) {
      float m = -INFINITY;
      for (int e = g * size; e < (g + 1) * size; ++e) m = fmaxf(m, s[e]);
      gs[g] = m;
    }
    __syncwarp();
    for (int g = lane; g < a.groups; g += 32) {
      int rank = 0;
      for (int o = 0; o < a.groups; ++o) rank += (gs[o] > gs[g] || (gs[o] == gs[g] && o < g)) ? 1 : 0;
      if (rank >= a.keep)
        for (int e = g * size; e < (g + 1) * size; ++e) s[e] = -1.0f;
    }
    __syncwarp();
  }
  float total = 0.f;
  for (int k = 0; k < a.top; ++k) {
    float bv = -2.0f;
    int bi = 0x7fffffff;
    for (int e = lane; e < a.experts; e += 32)
      if (s[e] > bv) { bv = s[e]; bi = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
    }
    if (bi >= a.experts) { bi = 0; bv = 0.f; }          // only when every score is NaN
    total += bv;
    if (lane == 0) {
      a.ids[row * a.top + k] = bi;
      a.weights[row * a.top + k] = bv;
      s[bi] = -2.0f;
    }
    __syncwarp();
  }
  const float norm = 1.0f / (total + 1e-20f);
  for (int k = lane; k < a.top; k += 32) a.weights[row * a.top + k] *= norm;
}

// One CTA.  counts -> first row of every expert (multiples of 128) -> tile list -> a row for every (token, k) pair.
// The order of the rows of one expert is not fixed; every row's result is independent of its place.
constexpr int kPlanThreads = 1024;
__global__ void __launch_bounds__(kPlanThreads) moe_plan_kernel(const mdb_moe_plan_args a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ int plan_smem[];
  int* count = plan_smem;              // [experts]
  int* first = plan_smem + a.experts;  // [experts]
  __shared__ int total_rows;
  for (int e = threadIdx.x; e < a.experts; e += kPlanThreads) count[e] = 0;
  __syncthreads();
  const int n = a.m * a.top;
  for (int i = threadIdx.x; i < n; i += kPlanThreads) {
    const int e = a.ids[i];
    if (e >= 0 && e < a.experts) atomicAdd(&count[e], 1);
  }
  __syncthreads();
  if (threadIdx.x < 32) {
    // exclusive prefix of the tile counts, 32 experts at a time
    int base = 0;
    for (int e0 = 0; e0 < a.experts; e0 += 32) {
      const int e = e0 + threadIdx.x;
      const int tiles = e < a.experts ? (count[e] + kMoeTileRows - 1) / kMoeTileRows : 0;
      int incl = tiles;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, incl, o);
        if (static_cast<int>(threadIdx.x) >= o) incl += v;
      }
      if (e < a.experts) {
        const int t0 = base + incl - tiles;
        first[e] = t0 * kMoeTileRows;
        for (int t = 0; t < tiles; ++t)
          if (t0 + t < a.max_tiles) a.tile_expert[t0 + t] = e;
      }
      base += __shfl_sync(0xffffffffu, incl, 31);
    }
    if (threadIdx.x == 0) {
      total_rows = base * kMoeTileRows;
      *a.num_tiles = base < a.max_tiles ? base : a.max_tiles;
    }
  }
  __syncthreads();
  const int cap = a.max_tiles * kMoeTileRows;
  for (int r = threadIdx.x; r < total_rows && r < cap; r += kPlanThreads) a.row_token[r] = -1;
  for (int e = threadIdx.x; e < a.experts; e += kPlanThreads) count[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += kPlanThreads) {
    const int e = a.ids[i];
    int slot = -1;
    if (e >= 0 && e < a.experts) {
      slot = first[e] + atomicAdd(&count[e], 1);
      if (slot < cap) a.row_token[slot] = i / a.top;
      else slot = -1;
    }
    a.slot[i] = slot;
  }
}

// (No __restrict__ on these pointers: a load the compiler may treat as invariant, like *num_tiles, moves above
// griddepcontrol.wait and then reads what the previous plan left.)
template <typename T>
__global__ void __launch_bounds__(128) moe_gather_kernel(const T* x, int64_t ldx, T* out, int width,
                                                         const int32_t* row_token,
                                                         const int32_t* num_tiles) {
  pdl_launch_dependents();
  pdl_wait();
  const int rows = *num_tiles * kMoeTileRows;
  const int chunks = width * static_cast<int>(sizeof(T)) / 16;
  for (int r = blockIdx.x; r < rows; r += gridDim.x) {
    const int t = row_token[r];
    if (t < 0) continue;                 // padding rows keep whatever they hold; nobody reads their results
    const uint4* src = reinterpret_cast<const uint4*>(x + static_cast<int64_t>(t) * ldx);
    uint4* dst = reinterpret_cast<uint4*>(out + static_cast<int64_t>(r) * width);
    for (int c = threadIdx.x; c < chunks; c += 128) dst[c] = src[c];
  }
}

}  // namespace mdb

using namespace mdb;

extern "C" {

int mdb_moe_route(const mdb_moe_route_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_moe_route_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.experts > 0 && a.top > 0 && a.groups > 0, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(a.experts % a.groups == 0 && a.keep > 0 && a.keep <= a.groups, MDB_ERR_ARG);
  MDB_REQUIRE(a.top <= a.keep * (a.experts / a.groups), MDB_ERR_ARG);
  MDB_REQUIRE(rows_present(a.logits) && a.ids && a.weights, MDB_ERR_ARG);
  const size_t smem = sizeof(float) * kRouteWarps * (a.experts + a.groups);
  MDB_REQUIRE(smem <= 48 * 1024, MDB_ERR_UNSUPPORTED);
  return mdb_launch(moe_route_kernel, dim3((a.m + kRouteWarps - 1) / kRouteWarps), dim3(kRouteWarps * 32), smem,
                    static_cast<cudaStream_t>(stream), a);
}

int mdb_moe_max_tiles(int m, int top, int experts) {
  if (m <= 0 || top <= 0 || experts <= 0) return 0;
  const int64_t pairs = static_cast<int64_t>(m) * top;
  const int64_t touched = pairs < experts ? pairs : experts;
  return static_cast<int>(touched + (pairs - touched) / kMoeTileRows);
}

int mdb_moe_plan(const mdb_moe_plan_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_moe_plan_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.experts > 0 && a.top > 0 && a.max_tiles > 0, MDB_ERR_ARG);
  MDB_REQUIRE(a.ids && a.slot && a.row_token && a.tile_expert && a.num_tiles, MDB_ERR_ARG);
  MDB_REQUIRE(a.experts <= 4096 && static_cast<int64_t>(a.m) * a.top < (1 << 30), MDB_ERR_UNSUPPORTED);
  return mdb_launch(moe_plan_kernel, dim3(1), dim3(kPlanThreads), sizeof(int) * 2 * a.experts,
                    static_cast<cudaStream_t>(stream), a);
}

int mdb_moe_gather(int dtype, const void* x, int64_t ldx, void* out, int width, const int32_t* row_token,
                   const int32_t* num_tiles, int max_tiles, mdb_stream_t stream) {
  MDB_REQUIRE(width > 0 && max_tiles >= 0 && ldx >= width, MDB_ERR_ARG);
  if (max_tiles == 0) return MDB_OK;
  MDB_REQUIRE(x && out && row_token && num_tiles, MDB_ERR_ARG);
  MDB_REQUIRE(width % 8 == 0 && ldx % 8 == 0 && mdb_aligned16(x) && mdb_aligned16(out), MDB_ERR_ALIGN);
  const int64_t rows = static_cast<int64_t>(max_tiles) * kMoeTileRows;
  const int grid = static_cast<int>(rows < 148 * 16 ? rows : 148 * 16);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == MDB_F32)
    return mdb_launch(moe_gather_kernel<float>, dim3(grid), dim3(128), 0, st, static_cast<const float*>(x), ldx,
                      static_cast<float*>(out), width, row_token, num_tiles);
  return mdb_launch(moe_gather_kernel<bf16>, dim3(grid), dim3(128), 0, st, static_cast<const bf16*>(x), ldx,
                    static_cast<bf16*>(out), width, row_token, num_tiles);
}

}  // extern "C"
