// Finishing a q/k/v projection whose heads the per-head kernel does not take:
//   - an RMSNorm over the whole query projection and one over the whole key projection
//     (gains of those sizes), or one per head, or none;
//   - key heads of size d and value heads of size dv that need not be equal;
//   - a layer that projects queries only (it reads another layer's keys and values);
//   - biases of the three projections, added here (in float32) rather than in the product;
//   - a query temperature: the query of position p times 1 + coef ln(floor((p + 1) / every) + 1);
//   - rotation of neighbouring pairs (2i, 2i + 1) instead of (i, i + rot_dim / 2);
//   - values mixed with another projection's values of the same token: v <- (1 - mix) v + mix other;
//   - several maps a head (differential attention): q and k have `maps` sub-heads of size d per head, each normed
//     (and rotated) by itself.  A key head's sub-heads lie side by side in its one row of D elements; a query
//     sub-head is a query head of its own whose d elements lie where its map's key lies, zeros elsewhere, so that
//     its score is its own map's alone and all maps share the one cached value.
// And what follows the attention of two maps: map_difference, out = rms(a1 - lambda a2) factor sigmoid(gate_h) over a
// head's dv values, from the attention's rows or, for decoded tokens, from the partials of their splits.
// Queries go to q_out [tokens, nq * D], keys and values into the cache pages
// [num_pages, 2, nkv, page_size, D]; D >= max(maps d, dv) is the one head size the attention
// kernels then work with, and the elements past d (dv) are written as zeros: a zero in a
// query or key adds nothing to a score, a zero value column gives a zero output column.
// One block per token.  Sums of squares are taken in float32 in a fixed order (a thread's
// elements ascending, lanes by xor-tree, warps ascending), so a token's bits do not depend
// on the batch.  Rotation: halves or neighbouring pairs of the first rot_dim elements of each head,
// products and sums rounded one by one as in rope.cuh.
#include "attention_fold.cuh"
#include "common.cuh"

namespace {

constexpr int THREADS = 256;

struct WideArgs {
  const void* qkv;          // [tokens, ld]: q (nq*d), then k (nkv*maps*d) and v (nkv*dv) if has_kv; nq counts sub-heads
  void* q_out;
  void* pages;
  const void* q_gain;       // scope 2: [nq*d]; scope 1: [d]; null: no norm
  const void* k_gain;
  const float* cos_table;   // [max_positions, rot_dim / 2]
  const float* sin_table;
  const int* positions;
  const int* token_req;
  const int* block_table;
  int64_t ld;
  int gain_bf16, table_stride, tokens, nq, nkv, d, dv, D, rot_dim, page_size, num_pages, max_positions;
  int scope;                // 0 none, 1 per head, 2 whole projection
  int has_kv, write_cache;
  float eps;
  const void* bias;         // null, or [ld]: the biases of q, k, v in the order of the projection's columns
  int bias_bf16;
  float temp_coef;          // query temperature (0: none)
  int temp_every;
  int interleaved;
  const void* v_other;      // null, or [tokens, v_other_ld]: values to mix into this layer's
  int64_t v_other_ld;
  const float* v_mix;       // one number
  int maps;                 // sub-heads of a head (1: none)
};

__device__ __forceinline__ float gain_at(const void* g, int bf16, int i) {
  return bf16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(g)[i])
              : reinterpret_cast<const float*>(g)[i];
}

// element i of a projection's row (at column `col0` of the whole row), with its bias
template <typename T>
__device__ __forceinline__ float biased_at(const WideArgs& a, const T* src, int col0, int i) {
  const float v = ls_to_float<T>(src[i]);
  return a.bias != nullptr ? v + gain_at(a.bias, a.bias_bf16, col0 + i) : v;
}

// sum of squares of src[0 .. n) by the whole block, fixed order
template <typename T>
__device__ float block_sumsq(const WideArgs& a, const T* src, int col0, int n, float* scratch) {
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += THREADS) {
    const float v = biased_at<T>(a, src, col0, i);
    ss = fmaf(v, v, ss);
  }
  return ls_block_sum(ss, scratch);
}

// One head of one token's queries or keys by one warp: d elements at src (column `col0` of the whole row), normed, rotated,
// times `factor`, written to dst[0 .. d).  `g0`: where the head's gain begins.
template <typename T>
__device__ __forceinline__ void finish_head(const WideArgs& a, const T* src, int col0, const void* gain, int g0, float rstd,
                                            const float* cs, const float* sn, float factor, T* dst) {
  const int d = a.d, half = a.rot_dim >> 1, lane = threadIdx.x & 31;
  if (a.scope == 1 && gain != nullptr) {
    float ss = 0.f;
    for (int i = lane; i < d; i += 32) {
      const float v = biased_at<T>(a, src, col0, i);
      ss = fmaf(v, v, ss);
    }
    rstd = 1.0f / sqrtf(ls_warp_sum(ss) / (float)d + a.eps);
  }
  auto normed = [&](int j) {
    float v = biased_at<T>(a, src, col0, j);
    if (gain != nullptr) v = __fmul_rn(__fmul_rn(v, rstd), gain_at(gain, a.gain_bf16, g0 + j));
    return v;
  };
  for (int i = lane; i < d; i += 32) {
    float out;
    if (i < a.rot_dim && a.interleaved) {
      const int r = i >> 1;
      const float lo = normed(2 * r), hi = normed(2 * r + 1);
      out = (i & 1) == 0 ? __fsub_rn(__fmul_rn(lo, cs[r]), __fmul_rn(hi, sn[r]))
                         : __fadd_rn(__fmul_rn(hi, cs[r]), __fmul_rn(lo, sn[r]));
    } else if (i < a.rot_dim) {
      if (i < half) {
        const float lo = normed(i), hi = normed(i + half);
        out = __fsub_rn(__fmul_rn(lo, cs[i]), __fmul_rn(hi, sn[i]));
      } else {
        const float lo = normed(i - half), hi = normed(i);
        out = __fadd_rn(__fmul_rn(hi, cs[i - half]), __fmul_rn(lo, sn[i - half]));
      }
    } else {
      out = normed(i);
    }
    if (factor != 1.0f) out = __fmul_rn(out, factor);
    dst[i] = ls_from_float<T>(out);
  }
}

// zeros in dst[from .. to), by one warp
template <typename T>
__device__ __forceinline__ void zero_span(T* dst, int from, int to) {
  for (int i = from + (int)(threadIdx.x & 31); i < to; i += 32) dst[i] = ls_from_float<T>(0.f);
}

// A block per token, a warp per head of q, then of k, then of v.
template <typename T>
__global__ void __launch_bounds__(THREADS) qkv_finish_kernel(WideArgs a, int* err) {
  __shared__ float scratch[32];
  ls_dependency_sync();
  const int t = blockIdx.x;
  const T* row = reinterpret_cast<const T*>(a.qkv) + (int64_t)t * a.ld;
  const int pos = a.positions[t];
  const int half = a.rot_dim >> 1;
  if (half > 0 && (pos < 0 || pos >= a.max_positions)) {
    if (threadIdx.x == 0) ls_record_fault(err, LS_DEV_POSITION_RANGE, t);
    return;
  }
  const float* cs = a.cos_table + (int64_t)pos * half;
  const float* sn = a.sin_table + (int64_t)pos * half;
  const int nk = a.nkv * a.maps;
  const bool writes = a.has_kv && a.write_cache;
  float q_rstd = 1.f, k_rstd = 1.f;
  if (a.scope == 2 && a.q_gain != nullptr)
    q_rstd = 1.0f / sqrtf(block_sumsq<T>(a, row, 0, a.nq * a.d, scratch) / (float)(a.nq * a.d) + a.eps);
  if (a.scope == 2 && a.k_gain != nullptr && writes) {
    __syncthreads();
    k_rstd = 1.0f / sqrtf(block_sumsq<T>(a, row + a.nq * a.d, a.nq * a.d, nk * a.d, scratch) / (float)(nk * a.d) + a.eps);
  }
  // where the token's keys and values go
  int page = -1, in_page = 0;
  if (writes) {
    const int req = a.token_req[t];
    page = a.block_table[(int64_t)req * a.table_stride + pos / a.page_size];
    in_page = pos % a.page_size;
    if (page < 0 || page >= a.num_pages) {
      if (threadIdx.x == 0) ls_record_fault(err, LS_DEV_PAGE_RANGE, t);
      page = -1;
    }
  }
  const float temperature =
      a.temp_coef != 0.f ? 1.0f + a.temp_coef * logf((float)((pos + 1) / a.temp_every + 1)) : 1.0f;
  const T* other = a.v_other != nullptr ? reinterpret_cast<const T*>(a.v_other) + (int64_t)t * a.v_other_ld : nullptr;
  const float mix = other != nullptr && page >= 0 ? *a.v_mix : 0.f;
  T* pages = reinterpret_cast<T*>(a.pages);
  const int tasks = a.nq + (page >= 0 ? nk + a.nkv : 0);
  for (int task = threadIdx.x >> 5; task < tasks; task += THREADS / 32) {
    if (task < a.nq) {
      // a query sub-head lies where its map's key lies, between zeros
      T* dst = reinterpret_cast<T*>(a.q_out) + ((int64_t)t * a.nq + task) * a.D;
      const int at = (task % a.maps) * a.d;
      finish_head<T>(a, row + task * a.d, task * a.d, a.q_gain, a.scope == 2 ? task * a.d : 0, q_rstd, cs, sn, temperature, dst + at);
      zero_span<T>(dst, 0, at);
      zero_span<T>(dst, at + a.d, a.D);
    } else if (task < a.nq + nk) {
      const int h = task - a.nq, slot = h / a.maps, map = h - slot * a.maps, col = task * a.d;
      T* dst = pages + ((((int64_t)page * 2 + 0) * a.nkv + slot) * a.page_size + in_page) * a.D;
      finish_head<T>(a, row + col, col, a.k_gain, a.scope == 2 ? h * a.d : 0, k_rstd, cs, sn, 1.0f, dst + map * a.d);
      if (map == a.maps - 1) zero_span<T>(dst, a.maps * a.d, a.D);
    } else {
      const int h = task - a.nq - nk, col = (a.nq + nk) * a.d;
      T* dst = pages + ((((int64_t)page * 2 + 1) * a.nkv + h) * a.page_size + in_page) * a.D;
      for (int i = threadIdx.x & 31; i < a.dv; i += 32) {
        float v = biased_at<T>(a, row + col, col, h * a.dv + i);
        if (other != nullptr) v = __fadd_rn(__fmul_rn(1.0f - mix, v), __fmul_rn(mix, ls_to_float<T>(other[h * a.dv + i])));
        dst[i] = ls_from_float<T>(v);
      }
      zero_span<T>(dst, a.dv, a.D);
    }
  }
}

// ---------------------------------------------------------------------------------------
// The difference of two maps: attention heads 2 h and 2 h + 1 are the maps of head h,
//   out[t, h, :] = u / sqrt(mean(u^2) + eps) * factor * sigmoid(gate[t, h]),  u = a_(2h) - lambda a_(2h+1),
// over the first dv elements of the attention's heads of D; float32 inside.  The sum of squares: a lane's
// elements c = lane, lane + 32, ... ascending, the lanes by an xor tree.
// ---------------------------------------------------------------------------------------
constexpr int DIFF_WARPS = 8;

template <typename T>
__device__ __forceinline__ float diff_gate(const T* __restrict__ gate, int64_t gate_ld, int t, int h, float factor) {
  return gate == nullptr ? factor : factor / (1.0f + expf(-ls_to_float<T>(gate[(int64_t)t * gate_ld + h])));
}

// rows of the attention's output: a warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(DIFF_WARPS * 32)
map_difference_kernel(const T* __restrict__ attn, const T* __restrict__ gate, int64_t gate_ld, T* __restrict__ out, int tokens,
                      int H, int D, int dv, float lambda, float factor, float eps) {
  ls_dependency_sync();
  const int64_t item = (int64_t)blockIdx.x * DIFF_WARPS + (threadIdx.x >> 5);
  if (item >= (int64_t)tokens * H) return;
  const int t = (int)(item / H), h = (int)(item - (int64_t)t * H), lane = threadIdx.x & 31;
  const T* a1 = attn + ((int64_t)t * 2 * H + 2 * h) * D;
  const T* a2 = a1 + D;
  float u[8], ss = 0.f;                                 // dv <= 256
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int c = lane + 32 * j;
    u[j] = c < dv ? fmaf(-lambda, ls_to_float<T>(a2[c]), ls_to_float<T>(a1[c])) : 0.f;
    ss = fmaf(u[j], u[j], ss);
  }
  ss = ls_warp_sum(ss);
  const float f = diff_gate<T>(gate, gate_ld, t, h, factor) / sqrtf(ss / (float)dv + eps);
  T* dst = out + ((int64_t)t * H + h) * dv;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int c = lane + 32 * j;
    if (c < dv) dst[c] = ls_from_float<T>(u[j] * f);
  }
}

// decoded tokens: a block per (combine item, head) folds both maps' splits first (each map's output is rounded to the
// engine's type, as the separate fold stores it: the same bits)
template <typename T>
__global__ void __launch_bounds__(256)
map_difference_fold_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml, const int* __restrict__ items,
                           const T* __restrict__ gate, int64_t gate_ld, T* __restrict__ out, int H, int D, int dv, float lambda,
                           float factor, float eps) {
  __shared__ float us[256];
  __shared__ float sum;
  ls_dependency_sync();
  const int* it = items + (int64_t)blockIdx.x * 4;
  const int tok = it[0], first = it[1], stride = it[2], n = it[3];
  if (n == 0) return;                                   // padding item of a recorded launch
  const int h = blockIdx.y, tid = threadIdx.x;
  for (int c = tid; c < dv; c += blockDim.x) {
    const float a1 = ls_fold_row(part_acc, part_ml, first, stride, n, 2 * H, 2 * h, D, c);
    const float a2 = ls_fold_row(part_acc, part_ml, first, stride, n, 2 * H, 2 * h + 1, D, c);
    us[c] = fmaf(-lambda, ls_to_float<T>(ls_from_float<T>(a2)), ls_to_float<T>(ls_from_float<T>(a1)));
  }
  __syncthreads();
  if (tid < 32) {
    float ss = 0.f;
    for (int j = 0; j < 8; ++j) {
      const int c = tid + 32 * j;
      const float v = c < dv ? us[c] : 0.f;
      ss = fmaf(v, v, ss);
    }
    ss = ls_warp_sum(ss);
    if (tid == 0) sum = ss;
  }
  __syncthreads();
  const float f = diff_gate<T>(gate, gate_ld, tok, h, factor) / sqrtf(sum / (float)dv + eps);
  for (int c = tid; c < dv; c += blockDim.x) out[((int64_t)tok * H + h) * dv + c] = ls_from_float<T>(us[c] * f);
}

}  // namespace

LS_API int ls_map_difference(const void* attn, const void* gate, int64_t gate_ld, void* out, int dtype, int tokens, int H, int D,
                             int dv, float lambda, float factor, float eps, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (H <= 0 || dv <= 0 || dv > 256 || D < dv || (gate != nullptr && gate_ld < H)) return LS_E_SIZE;
  const int64_t items = (int64_t)tokens * H;
  const dim3 grid((unsigned)((items + DIFF_WARPS - 1) / DIFF_WARPS)), block(DIFF_WARPS * 32);
  LS_COUNT(LS_K_MAP_DIFFERENCE);
  typedef __nv_bfloat16 bf16;
  if (dtype == LS_F32)
    ls_launch(map_difference_kernel<float>, grid, block, 0, stream, (const float*)attn, (const float*)gate, gate_ld, (float*)out,
              tokens, H, D, dv, lambda, factor, eps);
  else if (dtype == LS_BF16)
    ls_launch(map_difference_kernel<bf16>, grid, block, 0, stream, (const bf16*)attn, (const bf16*)gate, gate_ld, (bf16*)out,
              tokens, H, D, dv, lambda, factor, eps);
  else return LS_E_DTYPE;
  return ls_launch_status();
}

LS_API int ls_map_difference_fold(const float* part_acc, const float* part_ml, const int* items, int n_items, const void* gate,
                                  int64_t gate_ld, void* out, int dtype, int H, int D, int dv, float lambda, float factor,
                                  float eps, cudaStream_t stream) {
  if (n_items <= 0) return 0;
  if (H <= 0 || H > 65535 || dv <= 0 || dv > 256 || D < dv || (gate != nullptr && gate_ld < H)) return LS_E_SIZE;
  const dim3 grid(n_items, H), block(dv > 128 ? 256 : dv > 64 ? 128 : 64);
  LS_COUNT(LS_K_MAP_DIFFERENCE_FOLD);
  typedef __nv_bfloat16 bf16;
  if (dtype == LS_F32)
    ls_launch(map_difference_fold_kernel<float>, grid, block, 0, stream, part_acc, part_ml, items, (const float*)gate, gate_ld,
              (float*)out, H, D, dv, lambda, factor, eps);
  else if (dtype == LS_BF16)
    ls_launch(map_difference_fold_kernel<bf16>, grid, block, 0, stream, part_acc, part_ml, items, (const bf16*)gate, gate_ld,
              (bf16*)out, H, D, dv, lambda, factor, eps);
  else return LS_E_DTYPE;
  return ls_launch_status();
}

LS_API int ls_qkv_finish(const void* qkv, int64_t ld, void* q_out, void* pages, int dtype, const void* q_gain,
                         const void* k_gain, int gain_dtype, const float* cos_table, const float* sin_table,
                         const int* positions, const int* token_req, const int* block_table, int table_stride,
                         int tokens, int nq, int nkv, int d, int dv, int D, int rot_dim, int page_size,
                         int num_pages, int max_positions, float eps, int scope, int has_kv, int write_cache,
                         const void* bias, int bias_dtype, float temp_coef, int temp_every, int interleaved,
                         const void* v_other, int64_t v_other_ld, const float* v_mix, int maps, int* err, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (nq <= 0 || nkv <= 0 || d <= 0 || dv <= 0 || maps < 1 || D < (int64_t)maps * d || D < dv || scope < 0 || scope > 2 || nq % maps)
    return LS_E_SIZE;
  if (rot_dim < 0 || rot_dim > d || (rot_dim & 1)) return LS_E_SIZE;
  if (gain_dtype != LS_F32 && gain_dtype != LS_BF16) return LS_E_DTYPE;
  if (write_cache && (pages == nullptr || page_size <= 0)) return LS_E_SIZE;
  if (temp_coef != 0.f && temp_every <= 0) return LS_E_SIZE;
  if (bias != nullptr && bias_dtype != LS_F32 && bias_dtype != LS_BF16) return LS_E_DTYPE;
  if (v_other != nullptr && (v_mix == nullptr || !has_kv || v_other_ld < (int64_t)nkv * dv)) return LS_E_SIZE;
  WideArgs a;
  a.maps = maps; a.interleaved = interleaved; a.v_other = v_other; a.v_other_ld = v_other_ld; a.v_mix = v_mix;
  a.bias = bias; a.bias_bf16 = bias_dtype == LS_BF16 ? 1 : 0; a.temp_coef = temp_coef; a.temp_every = temp_every > 0 ? temp_every : 1;
  a.qkv = qkv; a.q_out = q_out; a.pages = pages; a.q_gain = q_gain; a.k_gain = k_gain;
  a.cos_table = cos_table; a.sin_table = sin_table; a.positions = positions; a.token_req = token_req;
  a.block_table = block_table; a.ld = ld; a.gain_bf16 = gain_dtype == LS_BF16 ? 1 : 0;
  a.table_stride = table_stride; a.tokens = tokens; a.nq = nq; a.nkv = nkv; a.d = d; a.dv = dv; a.D = D;
  a.rot_dim = rot_dim; a.page_size = page_size > 0 ? page_size : 1; a.num_pages = num_pages;
  a.max_positions = max_positions; a.scope = (q_gain == nullptr && k_gain == nullptr) ? 0 : scope;
  a.has_kv = has_kv; a.write_cache = write_cache; a.eps = eps;
  LS_COUNT(LS_K_QKV_FINISH);
  cudaError_t e;
  if (dtype == LS_F32) e = ls_launch(qkv_finish_kernel<float>, dim3(tokens), dim3(THREADS), 0, stream, a, err);
  else if (dtype == LS_BF16) e = ls_launch(qkv_finish_kernel<__nv_bfloat16>, dim3(tokens), dim3(THREADS), 0, stream, a, err);
  else return LS_E_DTYPE;
  if (e != cudaSuccess) return (int)e;
  return ls_launch_status();
}
