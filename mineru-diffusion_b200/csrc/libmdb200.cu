// Single translation unit of libmdb200.so: the kernels share one device status
// word and a few launch helpers, so the parts are included here in order
// rather than linked as relocatable device code.
#include "elementwise.cu"
#include "rows32.cu"
#include "attention.cu"
#include "sampler.cu"
#include "gemm_ws.cu"
#include "gemm_tc.cu"
#include "attention_tc.cu"
#include "api_linear.cu"
#include "moe.cu"
#include "gemm_f32.cu"
#include "api_gemm.cu"
#include "recurrent.cu"
#include "latent_attention.cu"
#include "window_attention.cu"
#include "chunk_scan.cu"
#include "tp_p2p.cu"
