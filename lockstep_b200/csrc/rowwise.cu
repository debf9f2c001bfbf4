// Row-wise kernels of designs that norm after a sublayer as well as before it:
//   - layer norm with a gain and an optional bias, (x - mean) rsqrt(var + eps) gain + bias, var the
//     mean of the squared deviations (rows may be gathered through row_index);
//   - the closing kernel of a sublayer: the RMS-normed results of mixers side by side, each with
//     a gain of its own, summed with one factor; optionally a layer norm of that sum; added to
//     the residual stream; optionally the layer norm of the new stream that the next sublayer reads;
//   - an embedding with a factor on the token's row and a second table indexed by a hash of the
//     token and the one before it, whose last row serves a sequence's first token;
//   - float32 rows written into some columns of a wider row of the engine's type; logits times a
//     factor, then capped with tanh;
//   - the gate of a token's own embedding in a layer: gelu(z) times some columns of the token's row of a table; for few
//     tokens with the product that makes z in the same kernel.
// All reductions run in float32 in an order fixed by the row's own width (a thread's elements
// ascending, the lanes by an xor tree, the warps ascending), so a row's result does not depend on the batch.
#include "common.cuh"

namespace {

constexpr int ROW_THREADS = 256;  // a block per row

template <typename TG>
__device__ __forceinline__ float gain_of(const TG* g, int i) { return ls_to_float<TG>(g[i]); }

// Sum over the block in a fixed order (lanes by xor tree, warps ascending); every thread gets it.  `scratch`: 32 floats.
__device__ __forceinline__ float row_sum(float v, float* scratch) {
  const float total = ls_block_sum(v, scratch);
  __syncthreads();                 // scratch is free for the next sum
  return total;
}

// a normed element times its gain, plus the bias where there is one
__device__ __forceinline__ float scaled(float u, float gain, bool biased, float bias) {
  return biased ? fmaf(u, gain, bias) : u * gain;
}

// (x - mean) rsqrt(var + eps) gain (+ bias) over float32 rows.  A thread takes the elements tid, tid + 256, ... of the row and
// keeps up to eight of them in registers between the passes (rows up to 2,048 wide are read once).
template <typename TG, typename TO>
__global__ void __launch_bounds__(ROW_THREADS)
layernorm_kernel(const float* __restrict__ x, const int* __restrict__ row_index, const TG* __restrict__ gain,
                 const TG* __restrict__ bias, TO* __restrict__ out, int rows, int width, int x_rows, float eps, int* err) {
  __shared__ float scratch[32];
  ls_dependency_sync();
  const int r = blockIdx.x, tid = threadIdx.x;
  int src_row = r;
  if (row_index != nullptr) {
    src_row = row_index[r];
    if (src_row < 0 || src_row >= x_rows) {
      if (tid == 0) ls_record_fault(err, LS_DEV_ROW_RANGE, r);
      src_row = 0;
    }
  }
  const float* row = x + (int64_t)src_row * width;
  constexpr int KEEP = 8;
  float v[KEEP];
#pragma unroll
  for (int j = 0; j < KEEP; ++j) v[j] = tid + j * ROW_THREADS < width ? row[tid + j * ROW_THREADS] : 0.f;
  float s = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) s += v[j];
  for (int i = tid + KEEP * ROW_THREADS; i < width; i += ROW_THREADS) s += row[i];
  const float mean = row_sum(s, scratch) / (float)width;
  float q = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const float d = tid + j * ROW_THREADS < width ? v[j] - mean : 0.f;
    q = fmaf(d, d, q);
  }
  for (int i = tid + KEEP * ROW_THREADS; i < width; i += ROW_THREADS) {
    const float d = row[i] - mean;
    q = fmaf(d, d, q);
  }
  const float rstd = 1.0f / sqrtf(row_sum(q, scratch) / (float)width + eps);
  TO* dst = out + (int64_t)r * width;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = tid + j * ROW_THREADS;
    if (i < width)
      dst[i] = ls_from_float<TO>(scaled((v[j] - mean) * rstd, gain_of<TG>(gain, i), bias != nullptr, bias != nullptr ? gain_of<TG>(bias, i) : 0.f));
  }
  for (int i = tid + KEEP * ROW_THREADS; i < width; i += ROW_THREADS)
    dst[i] = ls_from_float<TO>(scaled((row[i] - mean) * rstd, gain_of<TG>(gain, i), bias != nullptr, bias != nullptr ? gain_of<TG>(bias, i) : 0.f));
}

// residual += post(scale sum_b rms_b(x_b) gain_b), post = layer norm with post_gain (and post_bias), or nothing.  The
// merged row lies in shared memory between the passes.  With next_gain the layer norm of the new stream, with that gain
// (and next_bias), is written to next_out: sums and roundings are those of layernorm_kernel on the stored stream.
template <typename TO>
__global__ void __launch_bounds__(ROW_THREADS)
norm_merge_add_kernel(float* __restrict__ residual, const float* __restrict__ branches, int n, int64_t branch_stride,
                      const float* __restrict__ branch_gain, float scale, const float* __restrict__ post_gain,
                      const float* __restrict__ post_bias, const float* __restrict__ next_gain,
                      const float* __restrict__ next_bias, TO* __restrict__ next_out, int rows, int width, float eps_branch,
                      float eps_post, float eps_next) {
  extern __shared__ float merged[];                 // [width]
  __shared__ float scratch[32];
  ls_dependency_sync();
  const int r = blockIdx.x, tid = threadIdx.x;
  constexpr int MAX_N = 4;
  float rstd_b[MAX_N];
#pragma unroll
  for (int b = 0; b < MAX_N; ++b) {
    rstd_b[b] = 1.0f;
    if (b < n && branch_gain != nullptr) {
      const float* row = branches + b * branch_stride + (int64_t)r * width;
      float q = 0.f;
#pragma unroll 4
      for (int i = tid; i < width; i += ROW_THREADS) q = fmaf(row[i], row[i], q);
      rstd_b[b] = 1.0f / sqrtf(row_sum(q, scratch) / (float)width + eps_branch);
    }
  }
  float s = 0.f;
#pragma unroll 2
  for (int i = tid; i < width; i += ROW_THREADS) {
    float v = 0.f;
#pragma unroll
    for (int b = 0; b < MAX_N; ++b)
      if (b < n) {
        const float xb = branches[b * branch_stride + (int64_t)r * width + i];
        v += branch_gain != nullptr ? xb * rstd_b[b] * branch_gain[b * width + i] : xb;
      }
    v *= scale;
    merged[i] = v;                                  // (read back by this thread alone)
    s += v;
  }
  float* dst = residual + (int64_t)r * width;
  if (post_gain == nullptr) {
#pragma unroll 4
    for (int i = tid; i < width; i += ROW_THREADS) dst[i] = merged[i] = dst[i] + merged[i];
  } else {
    const float mean = row_sum(s, scratch) / (float)width;
    float q = 0.f;
    for (int i = tid; i < width; i += ROW_THREADS) {
      const float d = merged[i] - mean;
      q = fmaf(d, d, q);
    }
    const float rstd = 1.0f / sqrtf(row_sum(q, scratch) / (float)width + eps_post);
#pragma unroll 4
    for (int i = tid; i < width; i += ROW_THREADS) {
      const float u = (merged[i] - mean) * rstd;
      dst[i] = merged[i] = dst[i] + scaled(u, post_gain[i], post_bias != nullptr, post_bias != nullptr ? post_bias[i] : 0.f);
    }
  }
  if (next_gain == nullptr) return;
  s = 0.f;
  for (int i = tid; i < width; i += ROW_THREADS) s += merged[i];
  const float mean = row_sum(s, scratch) / (float)width;
  float q = 0.f;
  for (int i = tid; i < width; i += ROW_THREADS) {
    const float d = merged[i] - mean;
    q = fmaf(d, d, q);
  }
  const float rstd = 1.0f / sqrtf(row_sum(q, scratch) / (float)width + eps_next);
  TO* to = next_out + (int64_t)r * width;
#pragma unroll 4
  for (int i = tid; i < width; i += ROW_THREADS) {
    const float u = (merged[i] - mean) * rstd;
    to[i] = ls_from_float<TO>(scaled(u, next_gain[i], next_bias != nullptr, next_bias != nullptr ? next_bias[i] : 0.f));
  }
}

// The same for one result without a norm of its own (n = 1, no branch gain, scale 1) and rows of up to KEEP x 256
// elements: the row stays in registers, sums and roundings are those of norm_merge_add_kernel.
template <int KEEP, typename TO>
__global__ void __launch_bounds__(ROW_THREADS)
norm_add_kernel(float* __restrict__ residual, const float* __restrict__ x, const float* __restrict__ post_gain,
                const float* __restrict__ post_bias, const float* __restrict__ next_gain, const float* __restrict__ next_bias,
                TO* __restrict__ next_out, int width, float eps_post, float eps_next) {
  __shared__ float scratch[32];
  ls_dependency_sync();
  const int r = blockIdx.x, tid = threadIdx.x;
  const float* row = x + (int64_t)r * width;
  float* dst = residual + (int64_t)r * width;
  float v[KEEP], h[KEEP];
#pragma unroll
  for (int j = 0; j < KEEP; ++j) v[j] = tid + j * ROW_THREADS < width ? row[tid + j * ROW_THREADS] : 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) h[j] = tid + j * ROW_THREADS < width ? dst[tid + j * ROW_THREADS] : 0.f;
  auto moments = [&](const float (&u)[KEEP], float eps, float& mean, float& rstd) {
    float s = 0.f, q = 0.f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) s += u[j];
    mean = row_sum(s, scratch) / (float)width;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      const float d = tid + j * ROW_THREADS < width ? u[j] - mean : 0.f;
      q = fmaf(d, d, q);
    }
    rstd = 1.0f / sqrtf(row_sum(q, scratch) / (float)width + eps);
  };
  float mean, rstd;
  moments(v, eps_post, mean, rstd);
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = tid + j * ROW_THREADS;
    if (i < width) {
      const float u = (v[j] - mean) * rstd;
      dst[i] = h[j] = h[j] + scaled(u, post_gain[i], post_bias != nullptr, post_bias != nullptr ? post_bias[i] : 0.f);
    }
  }
  if (next_gain == nullptr) return;
  moments(h, eps_next, mean, rstd);
  TO* to = next_out + (int64_t)r * width;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = tid + j * ROW_THREADS;
    if (i < width) {
      const float u = (h[j] - mean) * rstd;
      to[i] = ls_from_float<TO>(scaled(u, next_gain[i], next_bias != nullptr, next_bias != nullptr ? next_bias[i] : 0.f));
    }
  }
}

// out[t] = table[id] factor + pairs[row(previous id, id)]
template <typename T>
__global__ void pair_embed_kernel(const int* __restrict__ ids, const int* __restrict__ token_slot,
                                  const int* __restrict__ carried, int64_t carried_stride, const T* __restrict__ table,
                                  const T* __restrict__ pairs, float* __restrict__ out, int width, int vocab, int buckets,
                                  long long mul_prev, long long mul_cur, float factor, int* err) {
  ls_dependency_sync();
  const int t = blockIdx.x;
  const int id = ids[t];
  float* dst = out + (int64_t)t * width;
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) ls_record_fault(err, LS_DEV_TOKEN_RANGE, t);
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = 0.f;
    return;
  }
  const T* src = table + (int64_t)id * width;
  if (pairs == nullptr) {
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = ls_to_float<T>(src[i]) * factor;
    return;
  }
  // the token before: the one in front of it in the step where that belongs to the same request, else what the
  // request's slot keeps (the last token of its last portion, plus one; zero: the request has none yet)
  const int slot = token_slot[t];
  long long prev = (t > 0 && token_slot[t - 1] == slot) ? (long long)ids[t - 1] : (long long)carried[slot * carried_stride] - 1;
  if (prev >= vocab) prev = -1;
  const long long row = prev < 0 ? buckets : (prev * mul_prev + (long long)id * mul_cur) % buckets;
  const T* pair = pairs + row * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x)
    dst[i] = fmaf(ls_to_float<T>(src[i]), factor, ls_to_float<T>(pair[i]));
}

// the last token of every request's portion, plus one, into the request's slot
__global__ void pair_carry_kernel(const int* __restrict__ ids, const int* __restrict__ token_slot,
                                  int* __restrict__ carried, int64_t carried_stride, int tokens) {
  ls_dependency_sync();
  const int t = blockIdx.x * blockDim.x + threadIdx.x;
  if (t >= tokens) return;
  const int slot = token_slot[t];
  if (t == tokens - 1 || token_slot[t + 1] != slot) carried[slot * carried_stride] = ids[t] + 1;
}

template <typename TO>
__global__ void rows_cast_kernel(const float* __restrict__ src, TO* __restrict__ dst, int64_t rows, int width, int64_t ld) {
  ls_dependency_sync();
  const int64_t n = rows * width;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t r = i / width;
    dst[r * ld + (i - r * width)] = ls_from_float<TO>(src[i]);
  }
}

__global__ void scale_cap_kernel(float* __restrict__ x, int64_t count, float factor, float cap) {
  ls_dependency_sync();
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < count; i += (int64_t)gridDim.x * blockDim.x) {
    const float v = x[i] * factor;
    x[i] = cap > 0.f ? cap * tanhf(v / cap) : v;
  }
}

// out[t, c] = gelu_tanh(z[t, c]) table[ids[t], at + c]
template <typename T>
__global__ void side_gate_kernel(const float* __restrict__ z, const int* __restrict__ ids, const T* __restrict__ table,
                                 int64_t table_ld, int at, int vocab, T* __restrict__ out, int64_t tokens, int dim, int* err) {
  ls_dependency_sync();
  const int64_t n = tokens * dim;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / dim;
    const int c = (int)(i - t * dim);
    const int id = ids[t];
    float v = 0.f;
    if (id < 0 || id >= vocab) {
      if (c == 0) ls_record_fault(err, LS_DEV_TOKEN_RANGE, (int)t);
    } else {
      v = ls_gelu_tanh(z[i]) * ls_to_float<T>(table[id * table_ld + at + c]);
    }
    out[i] = ls_from_float<T>(v);
  }
}

// The same with z[t, c] = h[t, :] . w[c, :] made here, for few tokens: a block has SIDE_ROWS rows of w and up to SIDE_TOKENS
// tokens, a thread every 128th piece of eight elements of all of them (a sum is a chain per thread over its pieces; the
// threads' sums are added sixteen at a time, then by an xor tree over eight lanes).
constexpr int SIDE_TOKENS = 8, SIDE_ROWS = 2, SIDE_THREADS = 128;

__global__ void __launch_bounds__(SIDE_THREADS)
side_gate_few_kernel(const float* __restrict__ h, const __nv_bfloat16* __restrict__ w, const int* __restrict__ ids,
                     const __nv_bfloat16* __restrict__ table, int64_t table_ld, int at, int vocab,
                     __nv_bfloat16* __restrict__ out, int tokens, int width, int dim, int* err) {
  __shared__ float sums[SIDE_ROWS * SIDE_TOKENS][SIDE_THREADS + 1];
  ls_dependency_trigger();
  const int tid = threadIdx.x, c0 = blockIdx.x * SIDE_ROWS, t0 = blockIdx.y * SIDE_TOKENS;
  const int left = tokens - t0 < SIDE_TOKENS ? tokens - t0 : SIDE_TOKENS;
  float acc[SIDE_ROWS][SIDE_TOKENS];
#pragma unroll
  for (int r = 0; r < SIDE_ROWS; ++r)
#pragma unroll
    for (int m = 0; m < SIDE_TOKENS; ++m) acc[r][m] = 0.f;
  ls_dependency_wait();
  for (int k = tid * 8; k < width; k += 8 * SIDE_THREADS) {
    // (rows past the last one are read again: the loads of a piece go out together)
    uint4 raw[SIDE_ROWS];
    float4 lo[SIDE_TOKENS], hi[SIDE_TOKENS];
#pragma unroll
    for (int r = 0; r < SIDE_ROWS; ++r)
      raw[r] = *reinterpret_cast<const uint4*>(w + (int64_t)(c0 + r < dim ? c0 + r : dim - 1) * width + k);
#pragma unroll
    for (int m = 0; m < SIDE_TOKENS; ++m) {
      const float4* src = reinterpret_cast<const float4*>(h + (int64_t)(t0 + (m < left ? m : left - 1)) * width + k);
      lo[m] = src[0];
      hi[m] = src[1];
    }
#pragma unroll
    for (int r = 0; r < SIDE_ROWS; ++r) {
      const float wf[8] = {__uint_as_float(raw[r].x << 16), __uint_as_float(raw[r].x & 0xffff0000u), __uint_as_float(raw[r].y << 16),
                           __uint_as_float(raw[r].y & 0xffff0000u), __uint_as_float(raw[r].z << 16),
                           __uint_as_float(raw[r].z & 0xffff0000u), __uint_as_float(raw[r].w << 16),
                           __uint_as_float(raw[r].w & 0xffff0000u)};
#pragma unroll
      for (int m = 0; m < SIDE_TOKENS; ++m) {
        float& s = acc[r][m];
        s = fmaf(lo[m].x, wf[0], s); s = fmaf(lo[m].y, wf[1], s); s = fmaf(lo[m].z, wf[2], s); s = fmaf(lo[m].w, wf[3], s);
        s = fmaf(hi[m].x, wf[4], s); s = fmaf(hi[m].y, wf[5], s); s = fmaf(hi[m].z, wf[6], s); s = fmaf(hi[m].w, wf[7], s);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < SIDE_ROWS; ++r)
#pragma unroll
    for (int m = 0; m < SIDE_TOKENS; ++m) sums[r * SIDE_TOKENS + m][tid] = acc[r][m];
  __syncthreads();
  // eight lanes an output
  const int o = tid >> 3, sub = tid & 7;
  static_assert(SIDE_THREADS == 8 * SIDE_ROWS * SIDE_TOKENS, "eight lanes an output");
  float z = 0.f;
#pragma unroll
  for (int i = 0; i < SIDE_THREADS / 8; ++i) z += sums[o][sub + 8 * i];
  z += __shfl_xor_sync(0xffffffffu, z, 4);
  z += __shfl_xor_sync(0xffffffffu, z, 2);
  z += __shfl_xor_sync(0xffffffffu, z, 1);
  const int c = c0 + o / SIDE_TOKENS, m = o % SIDE_TOKENS;
  if (sub == 0 && c < dim && m < left) {
    const int t = t0 + m, id = ids[t];
    float v = 0.f;
    if (id < 0 || id >= vocab) {
      if (c == 0) ls_record_fault(err, LS_DEV_TOKEN_RANGE, t);
    } else {
      v = ls_gelu_tanh(z) * __bfloat162float(table[id * table_ld + at + c]);
    }
    out[(int64_t)t * dim + c] = __float2bfloat16_rn(v);
  }
}

inline int blocks_for(int64_t n) { return (int)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16); }

}  // namespace

LS_API int ls_layernorm(const float* x, const int* row_index, const void* gain, const void* bias, int gain_dtype, void* out, int out_dtype,
                        int rows, int width, int x_rows, float eps, int* err, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (width <= 0) return LS_E_SIZE;
  const dim3 grid(rows), block(ROW_THREADS);
  LS_COUNT(LS_K_LAYERNORM);
#define LS_LN(TG, TO) \
  ls_launch(layernorm_kernel<TG, TO>, grid, block, 0, stream, x, row_index, (const TG*)gain, (const TG*)bias, (TO*)out, rows, width, x_rows, eps, err)
  if (gain_dtype == LS_F32 && out_dtype == LS_F32) LS_LN(float, float);
  else if (gain_dtype == LS_F32 && out_dtype == LS_BF16) LS_LN(float, __nv_bfloat16);
  else if (gain_dtype == LS_BF16 && out_dtype == LS_BF16) LS_LN(__nv_bfloat16, __nv_bfloat16);
  else if (gain_dtype == LS_BF16 && out_dtype == LS_F32) LS_LN(__nv_bfloat16, float);
  else return LS_E_DTYPE;
#undef LS_LN
  return ls_launch_status();
}

LS_API int ls_norm_merge_add(float* residual, const float* branches, int n, long long branch_stride, const float* branch_gain,
                             float scale, const float* post_gain, const float* post_bias, const float* next_gain,
                             const float* next_bias, void* next_out, int next_dtype, int rows, int width, float eps_branch,
                             float eps_post, float eps_next, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (width <= 0 || n < 1 || n > 4) return LS_E_SIZE;
  const size_t smem = sizeof(float) * (size_t)width;
  if (smem > 200 * 1024) return LS_E_SMEM;
  static size_t configured = 48 * 1024;
  if (next_gain != nullptr && (next_out == nullptr || (next_dtype != LS_F32 && next_dtype != LS_BF16))) return LS_E_DTYPE;
  if (smem > configured) {
    if (cudaFuncSetAttribute(norm_merge_add_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess ||
        cudaFuncSetAttribute(norm_merge_add_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return LS_E_SMEM;
    configured = smem;
  }
  if (next_gain != nullptr) LS_COUNT(LS_K_NORM_MERGE_NORM);
  else LS_COUNT(LS_K_NORM_MERGE_ADD);
  if (n == 1 && branch_gain == nullptr && scale == 1.0f && post_gain != nullptr && width <= 8 * ROW_THREADS) {
#define LS_NA(KEEP, TO)                                                                                                  \
  ls_launch(norm_add_kernel<KEEP, TO>, dim3(rows), dim3(ROW_THREADS), 0, stream, residual, branches, post_gain, post_bias, \
            next_gain, next_bias, (TO*)next_out, width, eps_post, eps_next)
    const bool f32 = next_gain == nullptr || next_dtype == LS_F32;
    if (width <= 4 * ROW_THREADS) {
      if (f32) LS_NA(4, float);
      else LS_NA(4, __nv_bfloat16);
    } else {
      if (f32) LS_NA(8, float);
      else LS_NA(8, __nv_bfloat16);
    }
#undef LS_NA
    return ls_launch_status();
  }
#define LS_NM(TO)                                                                                                       \
  ls_launch(norm_merge_add_kernel<TO>, dim3(rows), dim3(ROW_THREADS), smem, stream, residual, branches, n,              \
            (int64_t)branch_stride, branch_gain, scale, post_gain, post_bias, next_gain, next_bias, (TO*)next_out, rows, \
            width, eps_branch, eps_post, eps_next)
  if (next_gain == nullptr || next_dtype == LS_F32) LS_NM(float);
  else LS_NM(__nv_bfloat16);
#undef LS_NM
  return ls_launch_status();
}

LS_API int ls_pair_embed(const int* ids, const int* token_slot, int* carried, long long carried_stride, const void* table,
                         const void* pairs, int dtype, float* out, int tokens, int width, int vocab, int buckets,
                         long long mul_prev, long long mul_cur, float factor, int* err, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (pairs != nullptr && (buckets <= 0 || carried == nullptr || token_slot == nullptr)) return LS_E_SIZE;
  const int threads = width >= 1024 ? 256 : 128;
  LS_COUNT(LS_K_PAIR_EMBED);
  if (dtype == LS_F32)
    ls_launch(pair_embed_kernel<float>, tokens, threads, 0, stream, ids, token_slot, (const int*)carried, (int64_t)carried_stride,
              (const float*)table, (const float*)pairs, out, width, vocab, buckets, mul_prev, mul_cur, factor, err);
  else if (dtype == LS_BF16)
    ls_launch(pair_embed_kernel<__nv_bfloat16>, tokens, threads, 0, stream, ids, token_slot, (const int*)carried,
              (int64_t)carried_stride, (const __nv_bfloat16*)table, (const __nv_bfloat16*)pairs, out, width, vocab, buckets,
              mul_prev, mul_cur, factor, err);
  else
    return LS_E_DTYPE;
  if (ls_launch_status() != 0) return ls_launch_status();
  if (pairs != nullptr)
    ls_launch(pair_carry_kernel, dim3((tokens + 127) / 128), dim3(128), 0, stream, ids, token_slot, carried,
              (int64_t)carried_stride, tokens);
  return ls_launch_status();
}

LS_API int ls_rows_cast(const float* src, void* dst, int dst_dtype, long long rows, int width, long long ld, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (width <= 0 || ld < width) return LS_E_SIZE;
  LS_COUNT(LS_K_ROWS_CAST);
  if (dst_dtype == LS_F32) ls_launch(rows_cast_kernel<float>, blocks_for(rows * width), 256, 0, stream, src, (float*)dst, (int64_t)rows, width, (int64_t)ld);
  else if (dst_dtype == LS_BF16) ls_launch(rows_cast_kernel<__nv_bfloat16>, blocks_for(rows * width), 256, 0, stream, src, (__nv_bfloat16*)dst, (int64_t)rows, width, (int64_t)ld);
  else return LS_E_DTYPE;
  return ls_launch_status();
}

LS_API int ls_side_gate(const float* z, const int* ids, const void* table, long long table_ld, int at, int vocab, void* out,
                        int dtype, long long tokens, int dim, int* err, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (dim <= 0 || at < 0 || at + dim > table_ld || vocab <= 0) return LS_E_SIZE;
  LS_COUNT(LS_K_SIDE_GATE);
  if (dtype == LS_F32)
    ls_launch(side_gate_kernel<float>, blocks_for(tokens * dim), 256, 0, stream, z, ids, (const float*)table, (int64_t)table_ld,
              at, vocab, (float*)out, (int64_t)tokens, dim, err);
  else if (dtype == LS_BF16)
    ls_launch(side_gate_kernel<__nv_bfloat16>, blocks_for(tokens * dim), 256, 0, stream, z, ids, (const __nv_bfloat16*)table,
              (int64_t)table_ld, at, vocab, (__nv_bfloat16*)out, (int64_t)tokens, dim, err);
  else return LS_E_DTYPE;
  return ls_launch_status();
}

// bfloat16 weights, table and output; the width a multiple of 8, rows on 16-byte boundaries (else LS_E_ALIGN, nothing launched).
LS_API int ls_side_gate_few(const float* h, const void* w, const int* ids, const void* table, long long table_ld, int at,
                            int vocab, void* out, int tokens, int width, int dim, int* err, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (dim <= 0 || width <= 0 || at < 0 || at + dim > table_ld || vocab <= 0) return LS_E_SIZE;
  if (width % 8 || ((uintptr_t)h & 15) || ((uintptr_t)w & 15)) return LS_E_ALIGN;
  LS_COUNT(LS_K_SIDE_GATE_FEW);
  const dim3 grid((dim + SIDE_ROWS - 1) / SIDE_ROWS, (tokens + SIDE_TOKENS - 1) / SIDE_TOKENS);
  ls_launch(side_gate_few_kernel, grid, dim3(SIDE_THREADS), 0, stream, h, (const __nv_bfloat16*)w, ids,
            (const __nv_bfloat16*)table, (int64_t)table_ld, at, vocab, (__nv_bfloat16*)out, tokens, width, dim, err);
  return ls_launch_status();
}

LS_API int ls_scale_cap(float* x, long long count, float factor, float cap, cudaStream_t stream) {
  if (count <= 0) return 0;
  LS_COUNT(LS_K_SCALE_CAP);
  ls_launch(scale_cap_kernel, blocks_for(count), 256, 0, stream, x, (int64_t)count, factor, cap);
  return ls_launch_status();
}
