// What stands around the walk of mixers that carry a matrix state from token to token (the gated delta rule, an
// RWKV-style rule, gated linear attention, the matrix memory of an mLSTM; state_rules.cu): the list of a step's portions made on the device, short
// causal convolutions with their carried inputs, the token shift, the decays from the outputs
// of their low-rank maps (which run as products), and the gated per-head RMSNorm of the read-out.
//
// A step's token axis packs portions of several requests; a request appears once, so token t
// continues the portion of token t - 1 exactly when both have the same slot.  Everything a
// kernel needs to know about portions it takes from `token_slot` on the device, so a recorded
// step replays with other portions in the same buffers.
//
// All state and everything that enters a recurrence is float32.
#include "common.cuh"
#include "recurrent.cuh"

namespace {

// ---------------------------------------------------------------------------------------
// portions: out[0] = count, then (first token, tokens, slot) per portion, in token order
// ---------------------------------------------------------------------------------------
constexpr int PORTION_THREADS = 1024;

__global__ void __launch_bounds__(PORTION_THREADS) find_portions_kernel(const int* __restrict__ token_slot, int T,
                                                                       int* __restrict__ out, int cap, int* err) {
  __shared__ int warp_s[32], warp_e[32];
  __shared__ int base_s, base_e;
  ls_dependency_sync();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid == 0) base_s = base_e = 0;
  __syncthreads();
  for (int c0 = 0; c0 < T; c0 += PORTION_THREADS) {
    const int t = c0 + tid;
    int slot = 0;
    bool is_s = false, is_e = false;
    if (t < T) {
      slot = token_slot[t];
      is_s = t == 0 || token_slot[t - 1] != slot;
      is_e = t == T - 1 || token_slot[t + 1] != slot;
    }
    const unsigned bs = __ballot_sync(0xffffffffu, is_s), be = __ballot_sync(0xffffffffu, is_e);
    const unsigned below = (1u << lane) - 1u;
    if (lane == 0) {
      warp_s[warp] = __popc(bs);
      warp_e[warp] = __popc(be);
    }
    __syncthreads();
    int off_s = base_s, off_e = base_e, tot_s = 0, tot_e = 0;
    for (int w = 0; w < PORTION_THREADS / 32; ++w) {
      if (w < warp) {
        off_s += warp_s[w];
        off_e += warp_e[w];
      }
      tot_s += warp_s[w];
      tot_e += warp_e[w];
    }
    if (is_s) {
      const int p = off_s + __popc(bs & below);
      if (p < cap) {
        out[1 + 3 * p] = t;
        out[1 + 3 * p + 2] = slot;
      }
    }
    if (is_e) {
      const int p = off_e + __popc(be & below);
      if (p < cap) out[1 + 3 * p + 1] = t;     // the last token for now
    }
    __syncthreads();
    if (tid == 0) {
      base_s += tot_s;
      base_e += tot_e;
    }
    __syncthreads();
  }
  const int count = base_s;
  if (tid == 0) {
    out[0] = count < cap ? count : cap;
    if (count > cap) ls_record_fault(err, LS_DEV_ROW_RANGE, count);
  }
  __threadfence_block();
  __syncthreads();
  for (int p = tid; p < count && p < cap; p += PORTION_THREADS) out[1 + 3 * p + 1] = out[1 + 3 * p + 1] - out[1 + 3 * p] + 1;
}

// how many tokens before t lie in t's portion, at most `most`
__device__ __forceinline__ int tokens_before(const int* __restrict__ token_slot, int t, int most) {
  const int slot = token_slot[t];
  int m = 0;
  while (m < most && t - m - 1 >= 0 && token_slot[t - m - 1] == slot) ++m;
  return m;
}

// ---------------------------------------------------------------------------------------
// gated delta rule: everything between the projections and the recurrence
// ---------------------------------------------------------------------------------------
constexpr int PREP_THREADS = 256;

struct DeltaPrepArgs {
  const void* proj;        // [T, ld]: q (G dk) | k (G dk) | v (H dv) | beta (H) | ...
  int64_t ld;
  const float* conv_w;     // [C, taps], C = 2 G dk + H dv; the last tap is the current token's
  const float* dt_bias;    // [H dk]
  const float* a_log;      // [H]
  const float* state;      // per slot: S [H, dk, dv], then the last taps - 1 inputs of the convolution [taps - 1, C]
  int64_t state_stride;
  const int* token_slot;
  float* qkv;              // [T, C]: q (unit, scaled), k (unit), v, after convolution and silu
  float* decay;            // [T, H dk]: in, the output z of the decay's low-rank map; out, exp(-exp(A_log) softplus(z + dt_bias))
  float* beta;             // [T, H]
  int T, H, G, dk, dv, taps;
  float unit_eps;
  // null, or float32 [T, 2 H]: the logits of beta, then those of one decay per head (`decay` is [T, H] then, out only,
  // dt_bias [H]), instead of beta's logits in `proj` and a decay per channel
  const float* gates;
};

constexpr int PREP_WARPS = PREP_THREADS / 32;
constexpr int PREP_COLUMNS = 8;    // channels of a warp's segment that a lane has at most (heads up to 256)
constexpr int PREP_SEGMENT = 128;  // channels of a segment that is no head

// A warp has a segment of one token: a head of q or of k, 128 channels of v, 128 channels of the decay, or the token's
// numbers per head.
template <typename T>
__global__ void __launch_bounds__(PREP_THREADS) delta_prep_kernel(DeltaPrepArgs a, int v_segments) {
  ls_dependency_sync();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  int segment = blockIdx.y * PREP_WARPS + (threadIdx.x >> 5);
  const int Kd = a.G * a.dk, Vd = a.H * a.dv, C = 2 * Kd + Vd;
  const T* proj = reinterpret_cast<const T*>(a.proj);
  const T* row = proj + (int64_t)t * a.ld;
  if (segment < 2 * a.G + v_segments) {
    const int slot = a.token_slot[t];
    const int before = tokens_before(a.token_slot, t, a.taps - 1);
    const float* carried = a.state + (int64_t)slot * a.state_stride + (int64_t)a.H * a.dk * a.dv;
    const bool head = segment < 2 * a.G;
    const int first = head ? segment * a.dk : 2 * Kd + (segment - 2 * a.G) * PREP_SEGMENT;
    const int count = head ? a.dk : (C - first < PREP_SEGMENT ? C - first : PREP_SEGMENT);
    float v[PREP_COLUMNS];
    float ss = 0.f;
#pragma unroll
    for (int m = 0; m < PREP_COLUMNS; ++m) {
      const int i = lane + 32 * m, c = first + i;
      v[m] = 0.f;
      if (i >= count) continue;
      float acc = 0.f;
#pragma unroll 4
      for (int j = 0; j < a.taps; ++j) {
        const int back = a.taps - 1 - j;
        const float x = back <= before ? ls_to_float<T>(row[c - (int64_t)back * a.ld])
                                       : carried[(int64_t)(a.taps - 2 - (back - before - 1)) * C + c];
        acc = fmaf(a.conv_w[c * a.taps + j], x, acc);
      }
      v[m] = silu_f(acc);
      ss = fmaf(v[m], v[m], ss);
    }
    // q and k heads to unit length; q also by dk^(-1/2)
    float scale = 1.0f;
    if (head) scale = (1.0f / sqrtf(ls_warp_sum(ss) + a.unit_eps)) * (segment < a.G ? 1.0f / sqrtf((float)a.dk) : 1.0f);
    float* out = a.qkv + (int64_t)t * C + first;
#pragma unroll
    for (int m = 0; m < PREP_COLUMNS; ++m)
      if (lane + 32 * m < count) out[lane + 32 * m] = head ? v[m] * scale : v[m];
    return;
  }
  segment -= 2 * a.G + v_segments;
  if (segment == 0) {
    const float* z = a.gates + (int64_t)t * 2 * a.H;
    for (int h = lane; h < a.H; h += 32) {
      a.beta[(int64_t)t * a.H + h] = sigmoid_f(a.gates != nullptr ? z[h] : ls_to_float<T>(row[C + h]));
      if (a.gates != nullptr)
        a.decay[(int64_t)t * a.H + h] = expf(-expf(a.a_log[h]) * softplus_f(z[a.H + h] + a.dt_bias[h]));
    }
    return;
  }
  // a decay per channel
  const int channels = a.gates != nullptr ? 0 : a.H * a.dk;
  float* decay = a.decay + (int64_t)t * channels;
#pragma unroll
  for (int m = 0; m < PREP_SEGMENT / 32; ++m) {
    const int i = (segment - 1) * PREP_SEGMENT + lane + 32 * m;
    if (i < channels) decay[i] = expf(-expf(a.a_log[i / a.dk]) * softplus_f(decay[i] + a.dt_bias[i]));
  }
}

// z <- exp(-exp(z + bias[column])), element by element: a decay from its low-rank map's output
__global__ void __launch_bounds__(PREP_THREADS) double_exp_decay_kernel(float* __restrict__ z, const float* __restrict__ bias,
                                                                        int64_t count, int channels) {
  ls_dependency_sync();
  const int64_t i = (int64_t)blockIdx.x * PREP_THREADS + threadIdx.x;
  if (i < count) z[i] = expf(-expf(z[i] + bias[i % channels]));
}

// z <- sigmoid(z + bias[column])^(1 / tau), element by element, through its logarithm:
// exp(-softplus(-(z + bias)) / tau)
__global__ void __launch_bounds__(PREP_THREADS) sigmoid_power_decay_kernel(float* __restrict__ z, const float* __restrict__ bias,
                                                                           int64_t count, int channels, float inv_tau) {
  ls_dependency_sync();
  const int64_t i = (int64_t)blockIdx.x * PREP_THREADS + threadIdx.x;
  if (i < count) z[i] = expf(-softplus_f(-(z[i] + bias[i % channels])) * inv_tau);
}

// ---------------------------------------------------------------------------------------
// token shift: five mixes of a token with the one before it (the carried one at a portion's start)
// ---------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(PREP_THREADS) shift_mix_kernel(const T* __restrict__ x, const float* __restrict__ mu,
                                                                 const float* __restrict__ state, int64_t state_stride,
                                                                 int64_t prev_offset, const int* __restrict__ token_slot,
                                                                 T* __restrict__ out, int tokens, int width, int mixes) {
  ls_dependency_sync();
  const int t = blockIdx.x;
  const int slot = token_slot[t];
  const bool inside = t > 0 && token_slot[t - 1] == slot;
  const float* carried = state + (int64_t)slot * state_stride + prev_offset;
  for (int c = threadIdx.x; c < width; c += PREP_THREADS) {
    const float cur = ls_to_float<T>(x[(int64_t)t * width + c]);
    const float prev = inside ? ls_to_float<T>(x[(int64_t)(t - 1) * width + c]) : carried[c];
    const float diff = prev - cur;
    for (int s = 0; s < mixes; ++s)
      out[((int64_t)s * tokens + t) * width + c] = ls_from_float<T>(fmaf(diff, mu[s * width + c], cur));
  }
}

// x <- tanh(x), element by element
template <typename T>
__global__ void __launch_bounds__(PREP_THREADS) tanh_kernel(T* __restrict__ x, int64_t count) {
  ls_dependency_sync();
  const int64_t i = (int64_t)blockIdx.x * PREP_THREADS + threadIdx.x;
  if (i < count) x[i] = ls_from_float<T>(tanhf(ls_to_float<T>(x[i])));
}

// ---------------------------------------------------------------------------------------
// read-out: per-head RMSNorm, a gain, a gate
// ---------------------------------------------------------------------------------------
// out[t, h, j] = o[t, h, j] * rsqrt(mean_j o^2 + eps) * gain[shared ? j : h dv + j] * gate
//   gate_mode 0: gate_f32[t, h dv + j] as it is; 1: silu(gate_x[t, h dv + j]) from the engine's type;
//   2: sigmoid(gate_f32[t, h dv + j]); 3: sigmoid(gate_x[t, h dv + j])
// normalized: o's heads have two more elements, a and b, and o is first divided by max(|a|, b) + 1e-6
template <typename T>
__global__ void __launch_bounds__(PREP_THREADS) head_rms_gate_kernel(const float* __restrict__ o, const float* __restrict__ gain,
                                                                     const float* __restrict__ gate_f32,
                                                                     const T* __restrict__ gate_x, T* __restrict__ out,
                                                                     int H, int dv, int gain_shared, int gate_mode, float eps,
                                                                     int64_t gate_ld, int normalized) {
  ls_dependency_sync();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int h = warp; h < H; h += PREP_THREADS / 32) {
    const int64_t base = ((int64_t)t * H + h) * dv;
    const float* src = o + ((int64_t)t * H + h) * (normalized ? dv + 2 : dv);
    const float inv = normalized ? 1.0f / (fmaxf(fabsf(src[dv]), src[dv + 1]) + 1e-6f) : 1.0f;
    float ss = 0.f;
    for (int j = lane; j < dv; j += 32) {
      const float v = src[j] * inv;
      ss = fmaf(v, v, ss);
    }
    ss = ls_warp_sum(ss);
    const float rstd = 1.0f / sqrtf(ss / (float)dv + eps);
    for (int j = lane; j < dv; j += 32) {
      const float gt = gate_mode == 0 ? gate_f32[base + j]
                       : gate_mode == 2 ? sigmoid_f(gate_f32[base + j])
                       : gate_mode == 3 ? sigmoid_f(ls_to_float<T>(gate_x[(int64_t)t * gate_ld + h * dv + j]))
                                        : silu_f(ls_to_float<T>(gate_x[(int64_t)t * gate_ld + h * dv + j]));
      out[base + j] = ls_from_float<T>(src[j] * inv * rstd * gain[gain_shared ? j : h * dv + j] * gt);
    }
  }
}

}  // namespace

LS_API int ls_find_portions(const int* token_slot, int tokens, int* out, int cap, int* err, cudaStream_t stream) {
  if (tokens <= 0 || cap <= 0) return LS_E_SIZE;
  LS_COUNT(LS_K_FIND_PORTIONS);
  cudaError_t e = ls_launch(find_portions_kernel, dim3(1), dim3(PORTION_THREADS), 0, stream, token_slot, tokens, out, cap, err);
  if (e != cudaSuccess) return (int)e;
  return ls_launch_status();
}

LS_API int ls_delta_prep(const void* proj, int64_t ld, int dtype, const float* conv_w, const float* dt_bias,
                         const float* a_log, const float* state, int64_t state_stride, const int* token_slot,
                         float* qkv, float* decay, float* beta, const float* gates, int tokens, int H, int G, int dk,
                         int dv, int taps, float unit_eps, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0 || taps < 1 || taps > MAX_TAPS) return LS_E_SIZE;
  DeltaPrepArgs a;
  a.gates = gates;
  a.proj = proj; a.ld = ld; a.conv_w = conv_w; a.dt_bias = dt_bias; a.a_log = a_log; a.state = state;
  a.state_stride = state_stride; a.token_slot = token_slot; a.qkv = qkv; a.decay = decay; a.beta = beta; a.T = tokens;
  a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.taps = taps; a.unit_eps = unit_eps;
  if (dk > 32 * PREP_COLUMNS) return LS_E_SIZE;
  const int v_segments = (H * dv + PREP_SEGMENT - 1) / PREP_SEGMENT;
  const int segments = 2 * G + v_segments + 1 + (gates != nullptr ? 0 : (H * dk + PREP_SEGMENT - 1) / PREP_SEGMENT);
  const dim3 grid(tokens, (segments + PREP_WARPS - 1) / PREP_WARPS);
  if (grid.y > 65535) return LS_E_SIZE;
  LS_COUNT(LS_K_DELTA_PREP);
  cudaError_t e;
  if (dtype == LS_F32) e = ls_launch(delta_prep_kernel<float>, grid, dim3(PREP_THREADS), 0, stream, a, v_segments);
  else if (dtype == LS_BF16) e = ls_launch(delta_prep_kernel<__nv_bfloat16>, grid, dim3(PREP_THREADS), 0, stream, a, v_segments);
  else return LS_E_DTYPE;
  if (e != cudaSuccess) return (int)e;
  return ls_launch_status();
}

LS_API int ls_double_exp_decay(float* z, const float* bias, long long count, int channels, cudaStream_t stream) {
  if (count <= 0) return 0;
  if (channels <= 0) return LS_E_SIZE;
  LS_COUNT(LS_K_DOUBLE_EXP_DECAY);
  const dim3 grid((unsigned)((count + PREP_THREADS - 1) / PREP_THREADS));
  cudaError_t e = ls_launch(double_exp_decay_kernel, grid, dim3(PREP_THREADS), 0, stream, z, bias, (int64_t)count, channels);
  if (e != cudaSuccess) return (int)e;
  return ls_launch_status();
}

LS_API int ls_shift_mix(const void* x, int dtype, const float* mu, const float* state, int64_t state_stride,
                        int64_t prev_offset, const int* token_slot, void* out, int tokens, int width, int mixes,
                        cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (width <= 0 || mixes <= 0) return LS_E_SIZE;
  LS_COUNT(LS_K_SHIFT_MIX);
  cudaError_t e;
  if (dtype == LS_F32)
    e = ls_launch(shift_mix_kernel<float>, dim3(tokens), dim3(PREP_THREADS), 0, stream, (const float*)x, mu, state,
                  state_stride, prev_offset, token_slot, (float*)out, tokens, width, mixes);
  else if (dtype == LS_BF16)
    e = ls_launch(shift_mix_kernel<__nv_bfloat16>, dim3(tokens), dim3(PREP_THREADS), 0, stream, (const __nv_bfloat16*)x,
                  mu, state, state_stride, prev_offset, token_slot, (__nv_bfloat16*)out, tokens, width, mixes);
  else return LS_E_DTYPE;
  if (e != cudaSuccess) return (int)e;
  return ls_launch_status();
}

LS_API int ls_tanh_rows(void* x, int dtype, long long count, cudaStream_t stream) {
  if (count <= 0) return 0;
  LS_COUNT(LS_K_TANH);
  const dim3 grid((unsigned)((count + PREP_THREADS - 1) / PREP_THREADS));
  cudaError_t e;
  if (dtype == LS_F32) e = ls_launch(tanh_kernel<float>, grid, dim3(PREP_THREADS), 0, stream, (float*)x, (int64_t)count);
  else if (dtype == LS_BF16) e = ls_launch(tanh_kernel<__nv_bfloat16>, grid, dim3(PREP_THREADS), 0, stream, (__nv_bfloat16*)x, (int64_t)count);
  else return LS_E_DTYPE;
  if (e != cudaSuccess) return (int)e;
  return ls_launch_status();
}

LS_API int ls_sigmoid_power_decay(float* z, const float* bias, long long count, int channels, float tau, cudaStream_t stream) {
  if (count <= 0) return 0;
  if (channels <= 0 || !(tau > 0.f)) return LS_E_SIZE;
  LS_COUNT(LS_K_SIGMOID_POWER_DECAY);
  const dim3 grid((unsigned)((count + PREP_THREADS - 1) / PREP_THREADS));
  cudaError_t e = ls_launch(sigmoid_power_decay_kernel, grid, dim3(PREP_THREADS), 0, stream, z, bias, (int64_t)count, channels,
                            1.0f / tau);
  if (e != cudaSuccess) return (int)e;
  return ls_launch_status();
}

// gate_logit: the gate is the sigmoid of gate_f32 or of gate_x
LS_API int ls_head_rms_gate(const float* o, const float* gain, const float* gate_f32, const void* gate_x, void* out,
                            int dtype, int tokens, int H, int dv, int gain_shared, int gate_logit, float eps,
                            int64_t gate_ld, int normalized, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (H <= 0 || dv <= 0 || (gate_f32 == nullptr) == (gate_x == nullptr)) return LS_E_SIZE;
  const int mode = gate_f32 != nullptr ? (gate_logit ? 2 : 0) : (gate_logit ? 3 : 1);
  if (gate_ld <= 0) gate_ld = (int64_t)H * dv;       // the gate's rows lie one after the other
  LS_COUNT(LS_K_HEAD_RMS_GATE);
  cudaError_t e;
  if (dtype == LS_F32)
    e = ls_launch(head_rms_gate_kernel<float>, dim3(tokens), dim3(PREP_THREADS), 0, stream, o, gain, gate_f32,
                  (const float*)gate_x, (float*)out, H, dv, gain_shared, mode, eps, gate_ld, normalized);
  else if (dtype == LS_BF16)
    e = ls_launch(head_rms_gate_kernel<__nv_bfloat16>, dim3(tokens), dim3(PREP_THREADS), 0, stream, o, gain, gate_f32,
                  (const __nv_bfloat16*)gate_x, (__nv_bfloat16*)out, H, dv, gain_shared, mode, eps, gate_ld, normalized);
  else return LS_E_DTYPE;
  if (e != cudaSuccess) return (int)e;
  return ls_launch_status();
}

LS_API void ls_set_dependent_launch_seq(int on) { ls_dependent_launch = on ? 1 : 0; }
LS_API const char* ls_kernel_names_seq() { return LS_KERNEL_NAMES; }
LS_API int ls_kernel_launches_seq(unsigned long long* out, int n) {
  for (int i = 0; i < n && i < LS_K_COUNT; ++i) out[i] = ls_kernel_launches[i];
  return LS_K_COUNT;
}
LS_API const char* ls_constants_recurrent() {
  static char buf[256];
  static const LsConstant c[] = {{"recurrent.max_taps", MAX_TAPS}};
  return ls_format_constants(buf, sizeof buf, c, (int)(sizeof c / sizeof c[0]));
}
