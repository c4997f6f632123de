// y = x W^T in true fp32 (no tensor-core mode has a 24-bit significand): 64 x 64 tiles, 4 x 4 outputs per thread,
// operands through shared memory 16 k at a time.  Same three forms as the grouped tcgen05 kernel: plain, one weight
// per head (column blocks of x and y), one weight per expert (row tiles of 128).  GLU: gate rows and, n rows further, up rows
// side by side.  This serves the fp32 mode of the models that have one, where exactness matters more than speed.
#include "mdb_common.cuh"

namespace mdb {

constexpr int kF32Tile = 64, kF32K = 16;

template <bool GLU>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const mdb_gemm_args a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float xs[kF32K][kF32Tile + 4], ws[kF32K][kF32Tile + 4], us[GLU ? kF32K : 1][kF32Tile + 4];
  int64_t row0 = static_cast<int64_t>(blockIdx.y) * kF32Tile, w_row0 = 0;
  int x_col = 0, y_col = 0;
  if (a.form == MDB_GEMM_HEADS) {
    x_col = y_col = blockIdx.z;
    w_row0 = static_cast<int64_t>(blockIdx.z) * a.n;
    x_col *= a.k;
    y_col *= a.n;
  } else if (a.form == MDB_GEMM_EXPERTS) {
    const int tile = static_cast<int>(row0 / kMoeTileRows);
    if (tile >= *a.num_tiles) return;
    w_row0 = static_cast<int64_t>(a.tile_expert[tile]) * a.n;
  }
  const float* x = static_cast<const float*>(a.x);
  const float* w = static_cast<const float*>(a.w);
  const int n0 = blockIdx.x * kF32Tile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;      // loader: row of the tile, first of four k
  float acc[4][4] = {}, up[4][4] = {};
  for (int k0 = 0; k0 < a.k; k0 += kF32K) {
    float4 xv = make_float4(0.f, 0.f, 0.f, 0.f), wv = xv, uv = xv;
    if (row0 + lr < a.m) xv = *reinterpret_cast<const float4*>(x + (row0 + lr) * a.ldx + x_col + k0 + lk);
    if (n0 + lr < a.n) wv = *reinterpret_cast<const float4*>(w + (w_row0 + n0 + lr) * a.k + k0 + lk);
    if (GLU && n0 + lr < a.n) uv = *reinterpret_cast<const float4*>(w + (w_row0 + a.n + n0 + lr) * a.k + k0 + lk);
    __syncthreads();
    xs[lk][lr] = xv.x; xs[lk + 1][lr] = xv.y; xs[lk + 2][lr] = xv.z; xs[lk + 3][lr] = xv.w;
    ws[lk][lr] = wv.x; ws[lk + 1][lr] = wv.y; ws[lk + 2][lr] = wv.z; ws[lk + 3][lr] = wv.w;
    if (GLU) { us[GLU ? lk : 0][lr] = uv.x; us[GLU ? lk + 1 : 0][lr] = uv.y; us[GLU ? lk + 2 : 0][lr] = uv.z; us[GLU ? lk + 3 : 0][lr] = uv.w; }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kF32K; ++k) {
      float xr[4], wr[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { xr[i] = xs[k][ty * 4 + i]; wr[i] = ws[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          acc[i][j] = fmaf(xr[i], wr[j], acc[i][j]);
          if (GLU) up[i][j] = fmaf(xr[i], us[GLU ? k : 0][tx * 4 + j], up[i][j]);
        }
    }
  }
  float* y = static_cast<float*>(a.y);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int64_t row = row0 + ty * 4 + i;
    if (row >= a.m) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int col = n0 + tx * 4 + j;
      if (col >= a.n) continue;
      float v = acc[i][j];
      if (a.act == MDB_ACT_RELU2) { v = fmaxf(v, 0.f); v *= v; }
      if (a.act == MDB_ACT_SILU && col >= a.act_from) v /= 1.0f + expf(-v);
      if (GLU) v = fmaxf(v, 0.f) * up[i][j];
      y[row * a.ldy + y_col + col] = v;
    }
  }
}

static int gemm_f32_launch(const mdb_gemm_args& a, cudaStream_t st) {
  if (a.k % kF32K != 0) return MDB_ERR_UNSUPPORTED;
  const int64_t row_tiles = (static_cast<int64_t>(a.m) + kF32Tile - 1) / kF32Tile;
  if (row_tiles > 65535 || a.heads > 65535) return MDB_ERR_UNSUPPORTED;
  const dim3 grid((a.n + kF32Tile - 1) / kF32Tile, static_cast<int>(row_tiles), a.form == MDB_GEMM_HEADS ? a.heads : 1);
  if (a.act == MDB_ACT_RELU_GLU) return mdb_launch(gemm_f32_kernel<true>, grid, dim3(256), 0, st, a);
  return mdb_launch(gemm_f32_kernel<false>, grid, dim3(256), 0, st, a);
}

}  // namespace mdb
