// Shared declarations of the CUDA sources: element types, the device error
// word, and small conversion helpers.  Every launcher is a plain C function
// (loaded with ctypes) that takes raw device pointers and the stream to launch
// on, allocates nothing, and returns 0 or a negative LS_E_* code for arguments
// it refuses, or the positive cudaError_t of a failed launch.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>

#define LS_API extern "C" __attribute__((visibility("default")))

// element types of tensors handed to a launcher
enum { LS_F32 = 0, LS_BF16 = 1 };

// refusals of a launcher (returned, nothing is launched)
enum {
  LS_E_DTYPE = -1,     // unsupported element type combination
  LS_E_SIZE = -2,      // a size the kernel does not take
  LS_E_ALIGN = -3,     // a pointer or stride that is not aligned as required
  LS_E_SMEM = -4,      // needs more shared memory than the device offers
};

// faults a kernel records in the device error word (first fault wins); the host
// reads the word after the step and raises.
enum {
  LS_DEV_OK = 0,
  LS_DEV_TOKEN_RANGE = 1,   // token id outside the embedding table
  LS_DEV_PAGE_RANGE = 2,    // block table names a page outside the pool
  LS_DEV_POSITION_RANGE = 3,// position outside the rotary table
  LS_DEV_WAIT_TIMEOUT = 4,  // a bounded wait on a barrier ran out
  LS_DEV_ROW_RANGE = 5,     // a row index outside its tensor
};

__device__ __forceinline__ void ls_record_fault(int* err, int code, int detail) {
  if (err != nullptr) {
    if (atomicCAS(err, 0, code) == 0) err[1] = detail;
  }
}

// Launch constants that fix the order of a reduction are defined once, here or in the one
// source that uses them, and every source reports its own through ls_constants_<source>()
// as "name=value;..." so that a run can record the table it ran with.
#define LS_SPLIT 256         // keys of an attention split (fixed absolute positions)

struct LsConstant {
  const char* name;
  long long value;
};
static inline const char* ls_format_constants(char* buf, size_t size, const LsConstant* c, int count) {
  size_t at = 0;
  buf[0] = 0;
  for (int i = 0; i < count && at + 1 < size; ++i) {
    int n = snprintf(buf + at, size - at, "%s%s=%lld", i ? ";" : "", c[i].name, c[i].value);
    if (n < 0) break;
    at += (size_t)n;
  }
  return buf;
}

// Which kernels a process has launched (launcher calls, counted on the host): tests assert
// with it that the kernel they mean to check is the one that ran.
enum LsKernelId {
  LS_K_EMBED_GATHER = 0, LS_K_RMSNORM, LS_K_QK_NORM_ROPE, LS_K_QK_NORM_ROPE_WHOLE, LS_K_SILU_MUL,
  LS_K_GEMM_SIMT, LS_K_ATTENTION_TILE, LS_K_ATTENTION_DECODE, LS_K_ATTENTION_COMBINE, LS_K_ARGMAX,
  LS_K_SAMPLE, LS_K_GEMM_TC_FEW, LS_K_GEMM_TC_FEW_NORM, LS_K_GEMM_TC_FEW_QKV, LS_K_GEMM_TC_CLUSTER,
  LS_K_GEMM_TC_WALK, LS_K_GEMM_TC_ROWS, LS_K_GEMM_TC_ROWS_PAIR, LS_K_ATTENTION_DECODE_MMA,
  LS_K_ATTENTION_PREFILL_TC, LS_K_GEMM_SIMT_FEW, LS_K_GEMM_SIMT_MANY, LS_K_QKV_FINISH, LS_K_FIND_PORTIONS,
  LS_K_DELTA_PREP, LS_K_SHIFT_MIX, LS_K_DELTA_RULE, LS_K_WKV_RULE, LS_K_HEAD_RMS_GATE,
  LS_K_EXPERTS_ROUTE, LS_K_EXPERTS_PLAN, LS_K_EXPERTS_UP, LS_K_EXPERTS_DOWN, LS_K_EXPERTS_COMBINE,
  LS_K_EXPERTS_GATHER, LS_K_EXPERTS_UP_TC, LS_K_EXPERTS_DOWN_TC, LS_K_TANH, LS_K_DOUBLE_EXP_DECAY,
  LS_K_CLAMPED_GLU, LS_K_ROW_BIAS, LS_K_WEIGHTED_SUM, LS_K_GLA_RULE, LS_K_SIGMOID_POWER_DECAY, LS_K_LATENT_FINISH,
  LS_K_HEADS_PRODUCT, LS_K_GATED_SUM, LS_K_EXPERTS_MIX, LS_K_RMSNORM_SHIFT,
  LS_K_LAYERNORM, LS_K_NORM_MERGE_ADD, LS_K_PAIR_EMBED, LS_K_ROWS_CAST, LS_K_SCALE_CAP, LS_K_UNIT_GATES, LS_K_UNIT_SCAN,
  LS_K_ROTATE_ROWS, LS_K_DELTA_HEAD_RULE, LS_K_MLSTM_RULE, LS_K_SIDE_GATE, LS_K_SIDE_GATE_FEW,
  LS_K_MAP_DIFFERENCE, LS_K_MAP_DIFFERENCE_FOLD, LS_K_NORM_MERGE_NORM,
  LS_K_COUNT
};
#define LS_KERNEL_NAMES                                                                                  \
  "embed_gather,rmsnorm,qk_norm_rope_store,qk_norm_rope_store_whole,silu_mul,gemm_simt,attention_tile," \
  "attention_decode,attention_combine,argmax,sample,gemm_tc_few,gemm_tc_few_norm,gemm_tc_few_qkv,"      \
  "gemm_tc_cluster,gemm_tc_walk,gemm_tc_rows,gemm_tc_rows_pair,attention_decode_mma,attention_prefill_tc,"     \
  "gemm_simt_few,gemm_simt_many,qkv_finish,find_portions,delta_prep,shift_mix,delta_rule,"       \
  "wkv_rule,head_rms_gate,experts_route,experts_plan,experts_up,experts_down,experts_combine,"     \
  "experts_gather,experts_up_tc,experts_down_tc,tanh_rows,double_exp_decay,"                      \
  "clamped_glu,row_bias,weighted_sum,gla_rule,sigmoid_power_decay,latent_finish,heads_product,"  \
  "gated_sum,experts_mix,rmsnorm_shift,layernorm,norm_merge_add,pair_embed,rows_cast,scale_cap,unit_gates,"                 \
  "unit_scan,rotate_rows,delta_head_rule,mlstm_rule,side_gate,side_gate_few,"   \
  "map_difference,map_difference_fold,norm_merge_norm"
// one table per library: hidden, so that two libraries loaded into one process do not share it
__attribute__((visibility("hidden"))) inline unsigned long long ls_kernel_launches[LS_K_COUNT];
#define LS_COUNT(id) (++ls_kernel_launches[id])

template <typename T>
__device__ __forceinline__ float ls_to_float(T v);
template <>
__device__ __forceinline__ float ls_to_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ float ls_to_float<__nv_bfloat16>(__nv_bfloat16 v) {
  return __bfloat162float(v);
}

template <typename T>
__device__ __forceinline__ T ls_from_float(float v);
template <>
__device__ __forceinline__ float ls_from_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 ls_from_float<__nv_bfloat16>(float v) {
  return __float2bfloat16_rn(v);
}

__device__ __forceinline__ float ls_warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

__device__ __forceinline__ float ls_warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Sum over a thread block in a fixed order: lanes by xor-tree, then warps
// ascending.  `scratch` holds one float per warp (at most 32).  All threads
// get the result.
__device__ __forceinline__ float ls_block_sum(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  v = ls_warp_sum(v);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float total = 0.f;
  for (int w = 0; w < nwarps; ++w) total += scratch[w];
  return total;
}

// The first key position a query at `pos` reads: window > 0, the last `window` positions (a sliding
// window); window < 0, the positions of the query's own chunk of -window positions, chunks counted
// from position 0 of the sequence; 0, every earlier position.  It never falls as `pos` grows.
__host__ __device__ __forceinline__ int ls_first_key(int pos, int window) {
  if (window > 0) return pos - window + 1 > 0 ? pos - window + 1 : 0;
  if (window < 0) return pos - pos % (-window);
  return 0;
}

// Whether a query whose first key by the window is `lo` reads `key` (at or before it): the first `keep` keys of a
// sequence stay visible however far the window has moved on.
__host__ __device__ __forceinline__ bool ls_sees(int key, int lo, int keep) { return key >= lo || key < keep; }

// cap x tanh(score / cap) where a cap is given (cap > 0), else the score itself
__device__ __forceinline__ float ls_capped(float score, float cap) {
  return cap > 0.f ? cap * tanhf(score / cap) : score;
}

// the tanh form of gelu: 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3)))
__device__ __forceinline__ float ls_gelu_tanh(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// the square of relu
__device__ __forceinline__ float ls_relu_squared(float z) {
  const float r = fmaxf(z, 0.f);
  return r * r;
}

// Programmatic dependent launch: a kernel may be scheduled while its predecessor
// in the stream still runs.  Every kernel calls ls_dependency_sync() before it
// touches global memory: it lets the next kernel start being scheduled, then
// waits until the previous kernel has completed and its writes are visible.
__device__ __forceinline__ void ls_dependency_trigger() {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}
__device__ __forceinline__ void ls_dependency_wait() {
  asm volatile("griddepcontrol.wait;" ::: "memory");
}
__device__ __forceinline__ void ls_dependency_sync() {
  ls_dependency_trigger();
  ls_dependency_wait();
}

// one switch per library (set through ls_set_dependent_launch_<library>)
inline int ls_dependent_launch = 1;

template <typename... KArgs, typename... Args>
static inline cudaError_t ls_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                    cudaStream_t stream, Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = ls_dependent_launch ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

static inline int ls_launch_status() {
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : (int)e;
}
