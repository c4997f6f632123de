// C entry point of the linear layers of the fp32-residual decoders: one argument block for the plain, the per-head
// and the per-expert product, in bf16 (tcgen05 kernels) or true fp32.
#include "mdb_common.cuh"

using namespace mdb;

namespace {

int gemm_plain_bf16(const mdb_gemm_args& a, cudaStream_t st) {
  const bf16* x = static_cast<const bf16*>(a.x);
  const bf16* w = static_cast<const bf16*>(a.w);
  if (a.act == MDB_ACT_RELU_GLU) {
    MDB_REQUIRE(!a.y_f32, MDB_ERR_UNSUPPORTED);
    if (ws_supported(kWsSwiglu, a.m, 2 * a.n, a.k, a.ldx)) {
      WsArgs s = {};
      s.m = a.m; s.n = 2 * a.n; s.k = a.k; s.ksplit = 1;
      s.inter = a.n;
      s.glu_relu = 1;
      s.y = static_cast<bf16*>(a.y);
      s.ldy = a.ldy;
      return launch_ws<kWsSwiglu>(x, a.ldx, w, s, st);
    }
    MDB_REQUIRE(tc_supported(kTcSwiglu, a.m, a.n, a.k, a.ldx, a.ldy), MDB_ERR_UNSUPPORTED);
    TcArgs t = {};
    t.m = a.m; t.n = a.n; t.k = a.k; t.inter = a.n;
    t.act = a.act;
    t.y = static_cast<bf16*>(a.y);
    t.ldy = a.ldy;
    return launch_tc<kTcSwiglu>(x, a.ldx, w, 2 * a.n, t, st);
  }
  if (a.act == MDB_ACT_NONE && a.y_f32 && a.ldy == a.n && ws_supported(kWsPartial, a.m, a.n, a.k, a.ldx)) {
    // fp32 rows of a short step: one split-k slice of the streaming kernel
    WsArgs s = {};
    s.m = a.m; s.n = a.n; s.k = a.k; s.ksplit = 1;
    s.partials = static_cast<float*>(a.y);
    return launch_ws<kWsPartial>(x, a.ldx, w, s, st);
  }
  if (a.act == MDB_ACT_NONE && !a.y_f32 && a.n / kWsTileRows >= 64 && ws_supported(kWsBf16, a.m, a.n, a.k, a.ldx)) {
    WsArgs s = {};
    s.m = a.m; s.n = a.n; s.k = a.k; s.ksplit = 1;
    s.y = static_cast<bf16*>(a.y);
    s.ldy = a.ldy;
    return launch_ws<kWsBf16>(x, a.ldx, w, s, st);
  }
  MDB_REQUIRE(tc_supported(kTcBf16, a.m, a.n, a.k, a.ldx, a.ldy), MDB_ERR_UNSUPPORTED);
  TcArgs t = {};
  t.m = a.m; t.n = a.n; t.k = a.k;
  t.act = a.act;
  t.act_from = a.act_from;
  t.ldy = a.ldy;
  if (a.y_f32) t.y32 = static_cast<float*>(a.y);
  else t.y = static_cast<bf16*>(a.y);
  return launch_tc<kTcBf16>(x, a.ldx, w, a.n, t, st);
}

int gemm_group_bf16(const mdb_gemm_args& a, cudaStream_t st) {
  MDB_REQUIRE(a.k % kTcBK == 0 && a.n % 8 == 0 && a.ldx % 8 == 0 && a.ldy % 8 == 0, MDB_ERR_UNSUPPORTED);
  TcArgs t = {};
  t.m = a.m; t.n = a.n; t.k = a.k;
  t.act = a.act;
  t.ldy = a.ldy;
  if (a.y_f32) t.y32 = static_cast<float*>(a.y);
  else t.y = static_cast<bf16*>(a.y);
  if (a.form == MDB_GEMM_HEADS) {
    t.heads = a.heads;
    t.a_rows = a.m >= kTcBM ? kTcBM : (a.m + 15) / 16 * 16;
    return launch_tc_group(static_cast<const bf16*>(a.x), static_cast<int64_t>(a.heads) * a.k, a.ldx, static_cast<const bf16*>(a.w),
                           static_cast<int64_t>(a.heads) * a.n, t, st);
  }
  t.tile_expert = a.tile_expert;
  t.num_tiles = a.num_tiles;
  const int most = a.max_rows_per_expert;      // rows a tile can hold at most
  t.a_rows = most <= 0 || most >= kTcBM ? kTcBM : (most + 15) / 16 * 16;
  return launch_tc_group(static_cast<const bf16*>(a.x), a.k, a.ldx, static_cast<const bf16*>(a.w),
                         static_cast<int64_t>(a.experts) * a.n, t, st);
}

}  // namespace

extern "C" {

int mdb_gemm(const mdb_gemm_args* args, mdb_stream_t stream) {
  MDB_REQUIRE(args != nullptr, MDB_ERR_ARG);
  const mdb_gemm_args a = *args;
  MDB_REQUIRE(a.m >= 0 && a.n > 0 && a.k > 0, MDB_ERR_ARG);
  if (a.m == 0) return MDB_OK;
  MDB_REQUIRE(a.form >= MDB_GEMM_PLAIN && a.form <= MDB_GEMM_EXPERTS && a.act >= MDB_ACT_NONE && a.act <= MDB_ACT_SILU, MDB_ERR_ARG);
  MDB_REQUIRE(a.act < MDB_ACT_RELU_GLU || a.form == MDB_GEMM_PLAIN, MDB_ERR_UNSUPPORTED);
  MDB_REQUIRE(a.act_from >= 0 && a.act_from % 4 == 0 && (a.act == MDB_ACT_SILU || a.act_from == 0), MDB_ERR_ARG);
  MDB_REQUIRE(a.x && a.w && a.y, MDB_ERR_ARG);
  const int64_t groups = a.form == MDB_GEMM_HEADS ? a.heads : 1;
  MDB_REQUIRE(groups >= 1 && a.ldx >= groups * a.k && a.ldy >= groups * a.n, MDB_ERR_ARG);
  MDB_REQUIRE(a.form != MDB_GEMM_EXPERTS || (a.tile_expert && a.num_tiles && a.experts > 0 && a.m % kMoeTileRows == 0), MDB_ERR_ARG);
  MDB_REQUIRE(mdb_aligned16(a.x) && mdb_aligned16(a.w) && mdb_aligned16(a.y) && a.ldx % 8 == 0 && a.ldy % 4 == 0, MDB_ERR_ALIGN);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (a.dtype == MDB_F32) return gemm_f32_launch(a, st);
  return a.form == MDB_GEMM_PLAIN ? gemm_plain_bf16(a, st) : gemm_group_bf16(a, st);
}

}  // extern "C"
