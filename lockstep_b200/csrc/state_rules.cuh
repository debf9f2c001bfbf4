// The walk of a portion through a state rule: a matrix state per head and request slot, carried from token to token.
//
// A block has a portion, a head and some columns of the state.  One to four warps walk: a thread keeps ROWS key channels
// of one column in registers, L threads share a column.  Four more warps stage: they copy what the walk reads of every
// token (queries, keys, decays, values, the numbers of a token) into a ring of RING chunks of CHUNK tokens in shared
// memory, asynchronously (cp.async) and RING - 1 chunks ahead; float32 goes straight to its place, bfloat16 through a
// ring of its own from which the thread that copied it widens it one chunk ahead of the walk.  So neither the walk nor the
// staging waits for global memory.  UNIT tokens are walked in straight-line code: a token's read-out does not feed the
// state, so its sums run beside the next tokens' updates, and the exchange between the lanes of a column is made once per
// unit, for all its tokens, while the next unit is walked.
//
// A token's arithmetic is the same whatever portion or chunk it arrives in: states are walked token by token, a dot
// product over the key channels is four interleaved chains of fused multiply-adds per thread (channel r of the thread's
// run goes to chain r mod 4), added as (c0 + c1) + (c2 + c3), then an xor-tree over the lanes that share a column, the
// widest distance first.  (The exchange of a whole unit makes the same tree: a lane adds its partner's number to its own
// and keeps half of the tokens.)
#pragma once

#include <limits.h>

#include "common.cuh"
#include "recurrent.cuh"

namespace {

constexpr int ROWS = 16;           // key channels of a column that one thread keeps in registers
constexpr int CHUNK = 8;           // tokens staged in shared memory at a time
constexpr int STAGERS = 128;       // threads that stage
constexpr int MAX_WALK_WARPS = 4;
constexpr int UNIT = 4;            // tokens walked in straight-line code
constexpr int RING = 4;            // chunks in shared memory
constexpr int GATED = 32;          // mlstm: tokens whose gates are made at a time, by a warp of its own (a lane a token)
// what a staging thread copies of a chunk: pieces of 16 bytes of A, B, D, and pieces of 4 bytes of the rest (more than
// this, or rows that such pieces do not fit: the plain loader, with a ring of two)
constexpr int PIECES = 6;
constexpr int SINGLES = 3;
constexpr int MOST_SMEM = 160 * 1024;
// RULE_GLA: a decayed sum of outer products, S <- diag(decay_t) S + k_t v_t^T, o_t = out_scale S^T q_t
// RULE_DELTA_HEAD: RULE_DELTA with one decay per head.
// RULE_MLSTM: per head a log input gate i and a log forget gate f, from their logits z (i = cap tanh((z + b) / cap),
//   f = logsigmoid(cap tanh((z + b) / cap))), and a running maximum m from 0: m_t = max(f + m, i),
//   S <- exp(f + m - m_t) S + exp(i - m_t) k v^T, n <- the same with k alone, o = S^T q, n . q and exp(-m_t) read out.
//   n is one more column of S (a value that is always one), m one more row (a copy of it a column, so that every block
//   of columns reads and writes its own): the slot holds [H, dk + 1, dv + 1], the read-out [T, H, dv + 2].
enum { RULE_DELTA = 0, RULE_WKV = 1, RULE_GLA = 2, RULE_DELTA_HEAD = 3, RULE_MLSTM = 4 };

struct RuleArgs {
  const int* portions;     // from find_portions_kernel
  float* state;            // per slot: S [H, dk, dv] first
  int64_t state_stride;
  // delta: qkv float32 [T, 2 G dk + H dv], decay [T, H dk] or [T, H], beta [T, H]
  // wkv:   r, k, v [T, H dk] in the engine's type, decay [T, H dk], bonus [H dk]
  // gla, mlstm: q, k, v columns of rows of the engine's type, in_ld elements apart
  const void* in_a;        // delta: qkv; wkv: r; gla, mlstm: q
  const void* in_b;        // wkv, gla, mlstm: k
  const void* in_v;        // wkv, gla, mlstm: v
  const float* decay;
  const float* beta;       // delta
  const float* bonus;      // wkv
  float* out;              // [T, H dv] float32 (mlstm: [T, H (dv + 2)])
  // what else the state carries, brought up to date after the walk
  const void* carry_src;   // delta: the raw projection [T, ld] (its first C columns); wkv: the mixer's input [T, width]
  int64_t carry_ld;
  int carry_width;         // delta: C; wkv: width
  int carry_rows;          // delta: taps - 1; wkv: 1
  int H, G, dk, dv;
  int bf16;                // the engine's type is bfloat16 (else float32)
  int walkers;             // threads that walk
  int64_t in_ld;
  int pieces;              // everything can be copied in pieces (see PIECES)
  int raw_words;           // words of a chunk's bfloat16 rows on their way
  int numbers_at;          // mlstm: where in shared memory the gates' numbers lie
  float out_scale;         // gla, mlstm: factor on the read-out (the queries' scale)
  int64_t decay_ld;        // elements between two tokens' decays (H dk), or 0: one decay [H dk] for every token
  // mlstm: `decay` holds the gates' logits [T, 2 H] (all heads' i, then all heads' f), with these biases [2 H] and this cap
  const float* gate_bias;
  float gate_cap;
};

// One staged value's source: where token t's copy lies (p + t * stride), and its element type.
struct StageSrc {
  const char* p;
  int64_t stride;
  int kind;                // 0: nothing (zero), 1: float32, 2: bfloat16, 3: nothing (one)
};

__device__ __forceinline__ float engine_value(const void* p, int64_t i, int bf16) {
  return bf16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[i]) : reinterpret_cast<const float*>(p)[i];
}

// Two float32 lanes an instruction (sm_100: multiply and fused multiply-add on pairs of registers); every lane is rounded
// as the single instruction rounds it.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float x, float y) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& x, float& y) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(v));
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
// (c0 + c1) + (c2 + c3) of the chains in two pairs
__device__ __forceinline__ float sum_chains(f32x2 c01, f32x2 c23) {
  float c0, c1, c2, c3;
  unpack2(c01, c0, c1);
  unpack2(c23, c2, c3);
  return (c0 + c1) + (c2 + c3);
}

// The xor-tree over the L lanes of a column, for all tokens of a unit: after a step that halves, a lane holds the sums of
// the tokens its bit of `part` chooses.
template <int L>
__device__ __forceinline__ void fold_lanes(float (&o)[UNIT], int part) {
  int held = UNIT;
#pragma unroll
  for (int off = L >> 1; off > 0; off >>= 1) {
    if (held > 1) {
      held >>= 1;
      const bool upper = (part & off) != 0;
#pragma unroll
      for (int j = 0; j < UNIT / 2; ++j)
        if (j < held) {
          const float send = upper ? o[j] : o[j + held], keep = upper ? o[j + held] : o[j];
          o[j] = keep + __shfl_xor_sync(0xffffffffu, send, off);
        }
    } else {
      o[0] += __shfl_xor_sync(0xffffffffu, o[0], off);
    }
  }
}
__host__ __device__ constexpr int log2_of(int n) { return n <= 1 ? 0 : 1 + log2_of(n / 2); }

// This thread's channels of what a token brings.
struct TokenRows {
  ulonglong2 a[ROWS / 4], b[ROWS / 4], d[ROWS / 4];      // queries, keys, decays
};

// One token: the state's update, and this thread's share of the read-out.  `v`: the column's value; `beta`: of a delta
// rule; `keep`: the one decay of a rule that has one.
template <int RULE, int L>
__device__ __forceinline__ float advance(f32x2 (&S)[ROWS / 2], const f32x2* bonus, const TokenRows& t, float v, float beta,
                                         float keep) {
  constexpr bool DELTA = RULE == RULE_DELTA || RULE == RULE_DELTA_HEAD;
  constexpr bool ONE_DECAY = RULE == RULE_DELTA_HEAD || RULE == RULE_MLSTM;
  const f32x2 one_decay = pack2(keep, keep);
  f32x2 o01 = 0ull, o23 = 0ull;
  if constexpr (DELTA) {
    f32x2 d01 = 0ull, d23 = 0ull;
#pragma unroll
    for (int r = 0; r < ROWS / 4; ++r) {
      S[2 * r] = mul2(S[2 * r], ONE_DECAY ? one_decay : t.d[r].x); d01 = fma2(S[2 * r], t.b[r].x, d01);
      S[2 * r + 1] = mul2(S[2 * r + 1], ONE_DECAY ? one_decay : t.d[r].y); d23 = fma2(S[2 * r + 1], t.b[r].y, d23);
    }
    float dot = sum_chains(d01, d23);
#pragma unroll
    for (int off = L >> 1; off > 0; off >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, off);
    const float u = beta * (v - dot);
    const f32x2 u2 = pack2(u, u);
#pragma unroll
    for (int r = 0; r < ROWS / 4; ++r) {
      S[2 * r] = fma2(t.b[r].x, u2, S[2 * r]); o01 = fma2(S[2 * r], t.a[r].x, o01);
      S[2 * r + 1] = fma2(t.b[r].y, u2, S[2 * r + 1]); o23 = fma2(S[2 * r + 1], t.a[r].y, o23);
    }
  } else {
    const f32x2 v2 = pack2(v, v);
#pragma unroll
    for (int r = 0; r < ROWS / 4; ++r) {
      const f32x2 kx = mul2(t.b[r].x, v2), ky = mul2(t.b[r].y, v2);
      const f32x2 dx = ONE_DECAY ? one_decay : t.d[r].x, dy = ONE_DECAY ? one_decay : t.d[r].y;
      if constexpr (RULE == RULE_WKV) {
        o01 = fma2(t.a[r].x, fma2(bonus[2 * r], kx, S[2 * r]), o01); S[2 * r] = fma2(dx, S[2 * r], kx);
        o23 = fma2(t.a[r].y, fma2(bonus[2 * r + 1], ky, S[2 * r + 1]), o23); S[2 * r + 1] = fma2(dy, S[2 * r + 1], ky);
      } else {
        S[2 * r] = fma2(dx, S[2 * r], kx); o01 = fma2(t.a[r].x, S[2 * r], o01);
        S[2 * r + 1] = fma2(dy, S[2 * r + 1], ky); o23 = fma2(t.a[r].y, S[2 * r + 1], o23);
      }
    }
  }
  return sum_chains(o01, o23);
}

// The logs of an mlstm's input and forget gates from their logits.
__device__ __forceinline__ float log_input_gate(float z, float bias, float cap) { return cap * tanhf((z + bias) / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float bias, float cap) {
  return -softplus_f(-cap * tanhf((z + bias) / cap));
}

// The state of this thread's column, its channels part * ROWS ..., between memory and register pairs.
__device__ __forceinline__ void load_state(const float* state, int cols, int col, bool active, int part, int dk,
                                           f32x2 (&S)[ROWS / 2]) {
#pragma unroll
  for (int r = 0; r < ROWS / 2; ++r) {
    const int i = part * ROWS + 2 * r;
    S[r] = pack2((active && i < dk) ? state[(int64_t)i * cols + col] : 0.f,
                 (active && i + 1 < dk) ? state[(int64_t)(i + 1) * cols + col] : 0.f);
  }
}
__device__ __forceinline__ void store_state(float* state, int cols, int col, int part, int dk, const f32x2 (&S)[ROWS / 2]) {
#pragma unroll
  for (int r = 0; r < ROWS / 2; ++r) {
    const int i = part * ROWS + 2 * r;
    float x, y;
    unpack2(S[r], x, y);
    if (i < dk) state[(int64_t)i * cols + col] = x;
    if (i + 1 < dk) state[(int64_t)(i + 1) * cols + col] = y;
  }
}

// The rest of the state: the last inputs of a portion (its first token t0, n tokens), behind those that were carried.  All
// blocks of the portion share the channels.
__device__ __forceinline__ void carry_inputs(const RuleArgs& a, int slot, int t0, int n) {
  float* carried = a.state + (int64_t)slot * a.state_stride + (int64_t)a.H * a.dk * a.dv;
  const int rows = a.carry_rows, W = a.carry_width;
  const int block = blockIdx.y * gridDim.x + blockIdx.x, blocks = gridDim.x * gridDim.y;
  for (int c = block * blockDim.x + threadIdx.x; c < W; c += blocks * blockDim.x) {
    float keep[MAX_TAPS];
    for (int s = 0; s < rows; ++s) {
      const int from = n - rows + s;
      keep[s] = from >= 0 ? engine_value(a.carry_src, (int64_t)(t0 + from) * a.carry_ld + c, a.bf16)
                          : carried[(int64_t)(s + n) * W + c];
    }
    for (int s = 0; s < rows; ++s) carried[(int64_t)s * W + c] = keep[s];
  }
}

template <int RULE, int L>
__global__ void __launch_bounds__(STAGERS + 32 * MAX_WALK_WARPS + (RULE == RULE_MLSTM ? 32 : 0), 1)
rule_kernel(RuleArgs a) {
  extern __shared__ float smem[];
  ls_dependency_sync();
  const int p = blockIdx.z;          // (the slowest index: the blocks of the portions there are come first)
  if (p >= a.portions[0]) return;
  const int t0 = a.portions[1 + 3 * p], n = a.portions[1 + 3 * p + 1], slot = a.portions[1 + 3 * p + 2];
  constexpr bool DELTA = RULE == RULE_DELTA || RULE == RULE_DELTA_HEAD;
  constexpr bool ONE_DECAY = RULE == RULE_DELTA_HEAD || RULE == RULE_MLSTM;     // a decay per head, not per channel
  constexpr bool COLUMNS = RULE == RULE_GLA || RULE == RULE_MLSTM;              // q, k, v are columns of wider rows
  constexpr int MATS = ONE_DECAY ? 2 : 3;
  const int h = blockIdx.y, tid = threadIdx.x, CB = a.walkers / L;
  const int dk = a.dk, dv = a.dv;
  const int cols = RULE == RULE_MLSTM ? dv + 1 : dv, rows = RULE == RULE_MLSTM ? dk + 1 : dk;
  const int out_cols = RULE == RULE_MLSTM ? dv + 2 : dv;
  const int col0 = blockIdx.x * CB;
  const bool walker = tid < a.walkers;
  float* state = a.state + (int64_t)slot * a.state_stride + (int64_t)h * rows * cols;
  const int chunks = (n + CHUNK - 1) / CHUNK;

  // What is staged per token: A [dk] (q or r), B [dk] (k), D [dk] (decay), V [CB], and up to two numbers: beta and a
  // decay per head.  (mlstm: what is put in, what is kept and exp(-m) lie in a place of their own.)  In shared memory each of A, B, D
  // lies as L runs of ROWS channels, a run padded by four words: the lanes that share a column read 16 bytes each from
  // different banks, the lanes of other columns the same words.  Channels past dk stay zero (a zero key writes nothing).
  const int per_token = MATS * dk + CB + (RULE == RULE_DELTA_HEAD ? 2 : RULE == RULE_DELTA ? 1 : 0);
  constexpr int run = ROWS + 4, dkp = L * run;
  const int cbp = (CB + 3) & ~3;
  const int stride = MATS * dkp + cbp + 4;           // words of a token in shared memory
  const int v_at = MATS * dkp, n_at = v_at + cbp;    // where a token's values and its numbers lie
  const int ring = a.pieces ? RING : 2;
  auto buffer = [&](int c) { return smem + (c & (ring - 1)) * (CHUNK * stride); };      // where chunk c is staged
  auto meet = [&]() { asm volatile("bar.sync 1, %0;" ::"r"((int)blockDim.x) : "memory"); };

  if (dk < L * ROWS || a.pieces) {
    // zeros for the channels past dk and the columns past the head's; ones for the normalizer's column
    const int words = (chunks >= ring ? ring * CHUNK : n) * stride;
    const int one_at = RULE == RULE_MLSTM && dv >= col0 && dv < col0 + CB ? v_at + dv - col0 : -1;
    for (int e = tid; e < words; e += blockDim.x) smem[e] = RULE == RULE_MLSTM && e % stride == one_at ? 1.f : 0.f;
    meet();
  }

  // mlstm: the numbers of a token, two rounds of GATED tokens
  float4* const numbers = reinterpret_cast<float4*>(smem + a.numbers_at);
  if (walker) {
    const int cl = tid / L, part = tid % L, col = col0 + cl;
    const bool active = col < cols;
    // a thread keeps the key channels i = part * ROWS + r of its column, two to a register pair
    f32x2 S[ROWS / 2], bonus[ROWS / 2];
    load_state(state, cols, col, active, part, dk, S);
    if (RULE == RULE_WKV) load_state(a.bonus + h * dk, 1, 0, true, part, dk, bonus);
    float* out = a.out + ((int64_t)t0 * a.H + h) * out_cols + col;
    const int64_t out_step = (int64_t)a.H * out_cols;

    auto token = [&](const float* tok, const float4& gate) {
      const ulonglong2* A = reinterpret_cast<const ulonglong2*>(tok + part * run);
      const ulonglong2* B = reinterpret_cast<const ulonglong2*>(tok + dkp + part * run);
      const ulonglong2* D = reinterpret_cast<const ulonglong2*>(tok + 2 * dkp + part * run);
      TokenRows rows_of;
#pragma unroll
      for (int r = 0; r < ROWS / 4; ++r) {
        rows_of.a[r] = A[r];
        rows_of.b[r] = B[r];
        if (!ONE_DECAY) rows_of.d[r] = D[r];
      }
      const float v = RULE == RULE_MLSTM ? tok[v_at + cl] * gate.x : tok[v_at + cl];
      return advance<RULE, L>(S, bonus, rows_of, v, DELTA ? tok[n_at] : 0.f,
                              RULE == RULE_MLSTM ? gate.y : RULE == RULE_DELTA_HEAD ? tok[n_at + 1] : 0.f);
    };
    auto gate_of = [&](int t) {
      return RULE == RULE_MLSTM ? numbers[t & (2 * GATED - 1)] : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    auto write = [&](int t, float o, float floor) {
      if (COLUMNS) o *= a.out_scale;
      if (!active) return;
      float* dst = out + t * out_step;
      dst[0] = o;
      if (RULE == RULE_MLSTM && col == dv) dst[1] = floor;
    };
    constexpr int LOG = log2_of(L), HALVED = LOG < log2_of(UNIT) ? LOG : log2_of(UNIT), COUNT = UNIT >> HALVED;
    const int first = (part >> (LOG - HALVED)) * COUNT;      // which of a unit's tokens this lane writes
    const bool writes = (part & ((1 << (LOG - HALVED)) - 1)) == 0;
    // the unit before: its shares of the read-outs are exchanged and written while the next unit is walked
    float before[UNIT], floors[COUNT];
    int before_t = -1;
#pragma unroll
    for (int tt = 0; tt < UNIT; ++tt) before[tt] = 0.f;
#pragma unroll
    for (int j = 0; j < COUNT; ++j) floors[j] = 0.f;
    auto finish_unit = [&]() {                       // (without a branch in front: its sums run beside the walk's)
      fold_lanes<L>(before, part);
      if (writes && before_t >= 0) {
#pragma unroll
        for (int j = 0; j < COUNT; ++j) write(before_t + first + j, before[j], floors[j]);
      }
    };

    meet();                                          // the first chunk is staged
    for (int c = 0; c < chunks; ++c) {
      const float* buf = buffer(c);
      const int c0 = c * CHUNK;
      if (n - c0 >= CHUNK) {
#pragma unroll 1
        for (int u = 0; u < CHUNK; u += UNIT) {
          float o[UNIT];
#pragma unroll
          for (int tt = 0; tt < UNIT; ++tt) o[tt] = token(buf + (u + tt) * stride, gate_of(c0 + u + tt));
          finish_unit();
#pragma unroll
          for (int tt = 0; tt < UNIT; ++tt) before[tt] = o[tt];
          before_t = c0 + u;
#pragma unroll
          for (int j = 0; j < COUNT; ++j) floors[j] = RULE == RULE_MLSTM ? gate_of(before_t + first + j).z : 0.f;
        }
      } else {
        for (int tt = 0; tt < n - c0; ++tt) {
          const float4 gate = gate_of(c0 + tt);
          float o = token(buf + tt * stride, gate);
#pragma unroll
          for (int off = L >> 1; off > 0; off >>= 1) o += __shfl_xor_sync(0xffffffffu, o, off);
          if (part == 0) write(c0 + tt, o, gate.z);
        }
      }
      meet();
    }
    finish_unit();
    if (active) store_state(state, cols, col, part, dk, S);
    if (RULE == RULE_MLSTM) {
      meet();                                        // the running maximum after the last token
      if (active && part == 0) state[(int64_t)dk * cols + col] = numbers[0].x;
    }
  } else if (RULE == RULE_MLSTM && tid >= a.walkers + STAGERS) {
    // mlstm: the gates of GATED tokens (lane s has token s): both logits through the cap, then the running maximum token
    // by token (every lane walks them all, so that all know where the next round starts), then the three numbers
    const int lane = tid & 31, rounds = (n + GATED - 1) / GATED;
    constexpr int TURNS = GATED / CHUNK;             // chunks of a round
    const float bias_i = a.gate_bias[h], bias_f = a.gate_bias[a.H + h], cap = a.gate_cap;
    float m_run = state[(int64_t)dk * cols + (col0 < cols ? col0 : 0)];
    float z_i = 0.f, z_f = 0.f;
    auto ask = [&](int round) {
      const int t = round * GATED + lane;
      const float* z = a.decay + (int64_t)(t0 + (t < n ? t : n - 1)) * 2 * a.H + h;
      z_i = z[0];
      z_f = z[a.H];
    };
    auto make = [&](int round) {
      const int left = n - round * GATED;
      const float i_mine = log_input_gate(z_i, bias_i, cap), f_mine = log_forget_gate(z_f, bias_f, cap);
      float keep = 0.f, put = 0.f, floor = 0.f;
#pragma unroll
      for (int s = 0; s < GATED; ++s) {
        if (s >= left) break;
        const float li = __shfl_sync(0xffffffffu, i_mine, s), lf = __shfl_sync(0xffffffffu, f_mine, s);
        const float decayed = lf + m_run;
        const float m_new = fmaxf(decayed, li);
        if (s == lane) {
          keep = decayed - m_new;
          put = li - m_new;
          floor = -m_new;
        }
        m_run = m_new;
      }
      numbers[(round & 1) * GATED + lane] = make_float4(expf(put), expf(keep), expf(floor), 0.f);
    };
    ask(0);
    make(0);
    meet();
    for (int c = 0; c < chunks; ++c) {               // while chunk c is walked
      const int next = c / TURNS + 1;
      if (next < rounds && c % TURNS == 0) ask(next);
      if (next < rounds && c % TURNS == 1) make(next);
      meet();
    }
    if (lane == 0) numbers[0].x = m_run;
    meet();
  } else {
    const int st = tid - a.walkers;
    const int g = h / (a.H / a.G);
    const int Kd = a.G * dk, C = 2 * Kd + a.H * dv;
    const int engine_kind = a.bf16 ? 2 : 1, engine_size = a.bf16 ? 2 : 4;
    auto engine_at = [&](const void* base, int64_t i) { return reinterpret_cast<const char*>(base) + i * engine_size; };
    auto place = [&](int k) {                        // where fetched value k of a token lies
      if (k < MATS * dk) {
        const int which = k / dk, i = k - which * dk;
        return which * dkp + (i / ROWS) * run + (i % ROWS);
      }
      return k < MATS * dk + CB ? v_at + (k - MATS * dk) : n_at + (k - MATS * dk - CB);
    };
    auto source = [&](int k) {
      StageSrc s;
      s.p = nullptr; s.stride = 0; s.kind = 0;
      if (k >= per_token) return s;
      if (k < MATS * dk) {
        const int which = k / dk, i = k - which * dk;
        if (which == 2) {
          s.p = reinterpret_cast<const char*>(a.decay + h * dk + i);
          s.stride = a.decay_ld * 4;
          s.kind = 1;
        } else if (DELTA) {
          s.p = reinterpret_cast<const char*>(reinterpret_cast<const float*>(a.in_a) + which * Kd + g * dk + i);
          s.stride = (int64_t)C * 4;
          s.kind = 1;
        } else {
          s.p = engine_at(which == 0 ? a.in_a : a.in_b, h * dk + i);
          s.stride = (COLUMNS ? a.in_ld : (int64_t)a.H * dk) * engine_size;
          s.kind = engine_kind;
        }
      } else if (k < MATS * dk + CB) {
        const int j = col0 + (k - MATS * dk);
        if (RULE == RULE_MLSTM && j == dv) {
          s.kind = 3;                                // the normalizer's column: a value of one
        } else if (j < dv) {
          if (DELTA) {
            s.p = reinterpret_cast<const char*>(reinterpret_cast<const float*>(a.in_a) + 2 * Kd + h * dv + j);
            s.stride = (int64_t)C * 4;
            s.kind = 1;
          } else {
            s.p = engine_at(a.in_v, h * dv + j);
            s.stride = (COLUMNS ? a.in_ld : (int64_t)a.H * dv) * engine_size;
            s.kind = engine_kind;
          }
        }
      } else if (DELTA) {
        s.p = reinterpret_cast<const char*>((k == MATS * dk + CB ? a.beta : a.decay) + h);
        s.stride = (int64_t)a.H * 4;
        s.kind = 1;
      }
      return s;
    };
    if (a.pieces) {
      // Every thread copies the same places of every chunk.  16 bytes: of A and B (the engine's type, or float32), of D
      // (float32).  4 bytes: a float32 value or number, or two bfloat16 values.
      const bool wide = !DELTA && a.bf16;            // A, B and V are bfloat16: to the raw ring, widened later
      const int ab_values = wide ? 8 : 4, ab_pieces = dk / ab_values;
      const int token_pieces = 2 * ab_pieces + (MATS == 3 ? dk / 4 : 0);
      const int v_values = wide ? 2 : 1;
      const int v_cols = dv - col0 < CB ? (dv - col0 > 0 ? dv - col0 : 0) : CB;      // (the normalizer's column is no value)
      const int token_singles = v_cols / v_values + (per_token - MATS * dk - CB);
      float* const raw_ring = smem + RING * CHUNK * stride;
      const uint32_t ring_addr = (uint32_t)__cvta_generic_to_shared(smem);
      const uint32_t raw_addr = (uint32_t)__cvta_generic_to_shared(raw_ring);
      const int raw_token = dk + ((CB / 2 + 3) & ~3);        // words of a token in the raw ring: A, B, V (16-byte pieces)

      // a slot: where from (this chunk's), how far to the next chunk's, where to (words within a chunk's buffer or raw
      // buffer), the token within the chunk
      const char* from[PIECES + SINGLES];
      int64_t step[PIECES + SINGLES];
      int to[PIECES + SINGLES], token_of[PIECES + SINGLES], widen_to[PIECES + SINGLES];
#pragma unroll
      for (int m = 0; m < PIECES; ++m) {
        const int j = st + m * STAGERS;
        token_of[m] = INT_MAX;
        widen_to[m] = -1;
        if (j < token_pieces * CHUNK) {
          const int tt = j / token_pieces, e = j - tt * token_pieces;
          const bool is_d = e >= 2 * ab_pieces;
          const int which = is_d ? 2 : e / ab_pieces;
          const int i = is_d ? (e - 2 * ab_pieces) * 4 : (e - which * ab_pieces) * ab_values;
          const StageSrc src = source(which * dk + i);
          from[m] = src.p + (int64_t)(t0 + tt) * src.stride;
          step[m] = src.stride * CHUNK;
          token_of[m] = tt;
          to[m] = tt * stride + place(which * dk + i);
          if (wide && !is_d) {
            widen_to[m] = to[m];
            to[m] = tt * raw_token + (which * dk + i) / 2;
          }
        }
      }
#pragma unroll
      for (int m = PIECES; m < PIECES + SINGLES; ++m) {
        const int j = st + (m - PIECES) * STAGERS;
        token_of[m] = INT_MAX;
        widen_to[m] = -1;
        if (j < token_singles * CHUNK) {
          const int tt = j / token_singles, e = j - tt * token_singles;
          const bool is_v = e < v_cols / v_values;
          const int k = is_v ? MATS * dk + e * v_values : MATS * dk + CB + e - v_cols / v_values;
          const StageSrc src = source(k);
          from[m] = src.p + (int64_t)(t0 + tt) * src.stride;
          step[m] = src.stride * CHUNK;
          token_of[m] = tt;
          to[m] = tt * stride + place(k);
          if (wide && is_v) {
            widen_to[m] = to[m];
            to[m] = tt * raw_token + dk + e;
          }
        }
      }
      auto copy = [&](int c) {                       // start the copies of chunk c (called for 0, 1, 2, ... in turn)
        const int left = n - c * CHUNK;
        const uint32_t dst = ring_addr + (uint32_t)((c & (RING - 1)) * CHUNK * stride) * 4u;
        const uint32_t raw = raw_addr + (uint32_t)((c & (RING - 1)) * a.raw_words) * 4u;
#pragma unroll
        for (int m = 0; m < PIECES; ++m) {
          if (m * STAGERS >= token_pieces * CHUNK) break;
          if (token_of[m] < left)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((widen_to[m] >= 0 ? raw : dst) + (uint32_t)to[m] * 4u),
                         "l"(from[m]) : "memory");
          from[m] += step[m];
        }
#pragma unroll
        for (int m = PIECES; m < PIECES + SINGLES; ++m) {
          if ((m - PIECES) * STAGERS >= token_singles * CHUNK) break;
          if (token_of[m] < left)
            asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((widen_to[m] >= 0 ? raw : dst) + (uint32_t)to[m] * 4u),
                         "l"(from[m]) : "memory");
          from[m] += step[m];
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
      };
      // chunk c is there as far as this thread copied it (all but the two youngest groups): widen that
      auto finish = [&](int c) {
        asm volatile("cp.async.wait_group %0;" ::"n"(RING - 2) : "memory");
        const int left = n - c * CHUNK;
        float* buf = buffer(c);
        const float* raw = raw_ring + (c & (RING - 1)) * a.raw_words;
        if (wide) {
#pragma unroll
          for (int m = 0; m < PIECES; ++m) {
            if (m * STAGERS >= token_pieces * CHUNK) break;
            if (widen_to[m] < 0 || token_of[m] >= left) continue;
            const uint4 v = *reinterpret_cast<const uint4*>(raw + to[m]);
            float4* dst = reinterpret_cast<float4*>(buf + widen_to[m]);
            dst[0] = make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                                 __uint_as_float(v.y & 0xffff0000u));
            dst[1] = make_float4(__uint_as_float(v.z << 16), __uint_as_float(v.z & 0xffff0000u), __uint_as_float(v.w << 16),
                                 __uint_as_float(v.w & 0xffff0000u));
          }
#pragma unroll
          for (int m = PIECES; m < PIECES + SINGLES; ++m) {
            if ((m - PIECES) * STAGERS >= token_singles * CHUNK) break;
            if (widen_to[m] < 0 || token_of[m] >= left) continue;
            const uint32_t v = *reinterpret_cast<const uint32_t*>(raw + to[m]);
            *reinterpret_cast<float2*>(buf + widen_to[m]) = make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u));
          }
        }
      };
      for (int c = 0; c < RING - 1; ++c) copy(c);
      finish(0);
      meet();
      for (int c = 0; c < chunks; ++c) {             // while chunk c is walked
        copy(c + RING - 1);
        if (c + 1 < chunks) finish(c + 1);
        meet();
      }
    } else {
      auto load = [&](int c) {
        const int cn = n - c * CHUNK < CHUNK ? n - c * CHUNK : CHUNK;
        float* buf = buffer(c);
        for (int e = st; e < cn * per_token; e += STAGERS) {
          const int tt = e / per_token, k = e - tt * per_token;
          const StageSrc s = source(k);
          const char* src = s.p + (int64_t)(t0 + c * CHUNK + tt) * s.stride;
          buf[tt * stride + place(k)] = s.kind == 2 ? __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(src))
                                        : s.kind == 1 ? *reinterpret_cast<const float*>(src) : s.kind == 3 ? 1.f : 0.f;
        }
      };
      load(0);
      meet();
      for (int c = 0; c < chunks; ++c) {
        if (c + 1 < chunks) load(c + 1);
        meet();
      }
    }
    if (RULE == RULE_MLSTM) meet();
  }

  if (a.carry_rows > 0) carry_inputs(a, slot, t0, n);
}

// Steps of single tokens: every thread fetches what it needs of a token itself, beside its part of the state (nothing is
// staged and nobody is waited for).  Portions of several tokens are walked too, each token's fetch in front of it.
constexpr int STEP_THREADS = 128;

template <int RULE, int L>
__global__ void __launch_bounds__(STEP_THREADS, 4) rule_step_kernel(RuleArgs a) {
  ls_dependency_sync();
  const int p = blockIdx.z;
  if (p >= a.portions[0]) return;
  const int t0 = a.portions[1 + 3 * p], n = a.portions[1 + 3 * p + 1], slot = a.portions[1 + 3 * p + 2];
  constexpr bool DELTA = RULE == RULE_DELTA || RULE == RULE_DELTA_HEAD;
  constexpr bool ONE_DECAY = RULE == RULE_DELTA_HEAD || RULE == RULE_MLSTM;
  constexpr bool COLUMNS = RULE == RULE_GLA || RULE == RULE_MLSTM;
  const int h = blockIdx.y, tid = threadIdx.x, dk = a.dk, dv = a.dv;
  const int cols = RULE == RULE_MLSTM ? dv + 1 : dv, rows = RULE == RULE_MLSTM ? dk + 1 : dk;
  const int out_cols = RULE == RULE_MLSTM ? dv + 2 : dv;
  const int part = tid % L, col = blockIdx.x * (blockDim.x / L) + tid / L;
  const bool active = col < cols;
  const int g = h / (a.H / a.G), Kd = a.G * dk, C = 2 * Kd + a.H * dv;
  float* state = a.state + (int64_t)slot * a.state_stride + (int64_t)h * rows * cols;
  f32x2 S[ROWS / 2], bonus[ROWS / 2];
  load_state(state, cols, col, active, part, dk, S);
  if (RULE == RULE_WKV) load_state(a.bonus + h * dk, 1, 0, true, part, dk, bonus);
  float m_run = 0.f;
  if (RULE == RULE_MLSTM && active) m_run = state[(int64_t)dk * cols + col];

  const int wide = !DELTA && a.bf16;
  const bool whole = a.pieces && part * ROWS + ROWS <= dk;       // 16 channels on 16-byte boundaries
  // channels part * ROWS ... of a row that starts at element `at`, as register pairs (zeros past dk)
  auto channels = [&](const void* base, int64_t at, int bf16, ulonglong2 (&to)[ROWS / 4]) {
    at += part * ROWS;
    if (whole && bf16) {
      const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(base) + at);
#pragma unroll
      for (int r = 0; r < ROWS / 8; ++r) {
        const uint4 v = src[r];
        to[2 * r].x = pack2(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u));
        to[2 * r].y = pack2(__uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
        to[2 * r + 1].x = pack2(__uint_as_float(v.z << 16), __uint_as_float(v.z & 0xffff0000u));
        to[2 * r + 1].y = pack2(__uint_as_float(v.w << 16), __uint_as_float(v.w & 0xffff0000u));
      }
    } else if (whole) {
      const ulonglong2* src = reinterpret_cast<const ulonglong2*>(reinterpret_cast<const float*>(base) + at);
#pragma unroll
      for (int r = 0; r < ROWS / 4; ++r) to[r] = src[r];
    } else {
      auto value = [&](int i) { return part * ROWS + i < dk ? engine_value(base, at + i, bf16) : 0.f; };
#pragma unroll
      for (int r = 0; r < ROWS / 4; ++r) {
        to[r].x = pack2(value(4 * r), value(4 * r + 1));
        to[r].y = pack2(value(4 * r + 2), value(4 * r + 3));
      }
    }
  };
  for (int tt = 0; tt < n; ++tt) {
    const int64_t t = t0 + tt;
    TokenRows rows_of;
    float v = 0.f, beta = 0.f, keep = 0.f, floor = 0.f;
    if constexpr (DELTA) {
      channels(a.in_a, t * C + g * dk, 0, rows_of.a);
      channels(a.in_a, t * C + Kd + g * dk, 0, rows_of.b);
      if (active) v = reinterpret_cast<const float*>(a.in_a)[t * C + 2 * Kd + h * dv + col];
      beta = a.beta[t * a.H + h];
      if (ONE_DECAY) keep = a.decay[t * a.H + h];
    } else {
      const int64_t k_ld = COLUMNS ? a.in_ld : (int64_t)a.H * dk, v_ld = COLUMNS ? a.in_ld : (int64_t)a.H * dv;
      channels(a.in_a, t * k_ld + h * dk, wide, rows_of.a);
      channels(a.in_b, t * k_ld + h * dk, wide, rows_of.b);
      if (RULE == RULE_MLSTM && col == dv) v = 1.f;
      else if (active) v = engine_value(a.in_v, t * v_ld + h * dv + col, wide);
    }
    if (!ONE_DECAY) channels(a.decay, t * a.decay_ld + h * dk, 0, rows_of.d);
    if constexpr (RULE == RULE_MLSTM) {
      const float* z = a.decay + t * 2 * a.H + h;
      const float li = log_input_gate(z[0], a.gate_bias[h], a.gate_cap);
      const float decayed = log_forget_gate(z[a.H], a.gate_bias[a.H + h], a.gate_cap) + m_run;
      m_run = fmaxf(decayed, li);
      v *= expf(li - m_run);
      keep = expf(decayed - m_run);
      floor = expf(-m_run);
    }
    float o = advance<RULE, L>(S, bonus, rows_of, v, beta, keep);
#pragma unroll
    for (int off = L >> 1; off > 0; off >>= 1) o += __shfl_xor_sync(0xffffffffu, o, off);
    if (COLUMNS) o *= a.out_scale;
    if (active && part == 0) {
      float* dst = a.out + (t * a.H + h) * out_cols + col;
      dst[0] = o;
      if (RULE == RULE_MLSTM && col == dv) dst[1] = floor;
    }
  }
  if (active) {
    store_state(state, cols, col, part, dk, S);
    if (RULE == RULE_MLSTM && part == 0) state[(int64_t)dk * cols + col] = m_run;
  }
  if (a.carry_rows > 0) carry_inputs(a, slot, t0, n);
}

template <int RULE, int L>
int launch_step(RuleArgs& a, int max_portions, cudaStream_t stream) {
  const int cols = RULE == RULE_MLSTM ? a.dv + 1 : a.dv;
  int threads = STEP_THREADS;
  while (threads > 32 && (threads / 2) / L >= cols) threads /= 2;
  const int cb = threads / L;
  cudaError_t e = ls_launch(rule_step_kernel<RULE, L>, dim3((cols + cb - 1) / cb, a.H, max_portions), dim3(threads), 0, stream, a);
  if (e != cudaSuccess) return (int)e;
  return ls_launch_status();
}

template <int RULE, int L>
int launch_walk(RuleArgs& a, int max_portions, cudaStream_t stream) {
  const int cols = RULE == RULE_MLSTM ? a.dv + 1 : a.dv;
  const int per_warp = 32 / L, needed = (cols + per_warp - 1) / per_warp;      // columns of a warp, warps of a head
  // Walking warps a block: few blocks have many tokens each, so as few warps a block as give every SM one block (a walk is
  // then issued without a rival)
  int warps = 1;
  while (warps < MAX_WALK_WARPS && warps < needed && (long long)a.H * ((needed + warps - 1) / warps) > 148) warps *= 2;
  // (a chunk's values of that many columns are what the staging threads copy ahead)
  while (warps > 1 && (32 * warps / L + 2) * CHUNK > SINGLES * STAGERS) warps /= 2;
  a.walkers = 32 * warps;
  const int cb = a.walkers / L;
  const int mats = RULE == RULE_DELTA_HEAD || RULE == RULE_MLSTM ? 2 : 3;
  // chunks of CHUNK tokens, a token as the kernel lays it out, and (pieces of bfloat16, gates' logits) what is on its way
  const size_t chunk_words = (size_t)CHUNK * (mats * L * (ROWS + 4) + ((cb + 3) & ~3) + 4);
  const bool wide = (RULE == RULE_WKV || RULE == RULE_GLA || RULE == RULE_MLSTM) && a.bf16;
  a.raw_words = wide ? CHUNK * (a.dk + ((cb / 2 + 3) & ~3)) : 0;
  const int pieces = 2 * a.dk / (wide ? 8 : 4) + (mats == 3 ? a.dk / 4 : 0);
  const size_t ring_bytes = sizeof(float) * RING * (chunk_words + a.raw_words);
  if (pieces * CHUNK > PIECES * STAGERS || ring_bytes > MOST_SMEM - 4096 || (wide && (cb % 2 || a.dv % 2))) a.pieces = 0;
  size_t smem = a.pieces ? ring_bytes : sizeof(float) * 2 * chunk_words;
  a.numbers_at = (int)(smem / sizeof(float));
  if (RULE == RULE_MLSTM) smem += sizeof(float4) * 2 * GATED;
  if (smem > MOST_SMEM) return LS_E_SMEM;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(rule_kernel<RULE, L>, cudaFuncAttributeMaxDynamicSharedMemorySize, MOST_SMEM) != cudaSuccess)
      return LS_E_SMEM;
    configured = true;
  }
  const dim3 grid((cols + cb - 1) / cb, a.H, max_portions);
  cudaError_t e = ls_launch(rule_kernel<RULE, L>, grid, dim3(a.walkers + STAGERS + (RULE == RULE_MLSTM ? 32 : 0)), smem, stream, a);
  if (e != cudaSuccess) return (int)e;
  return ls_launch_status();
}

template <int RULE, int L>
int launch(RuleArgs& a, int tokens, int max_portions, cudaStream_t stream) {
  return tokens <= max_portions ? launch_step<RULE, L>(a, max_portions, stream) : launch_walk<RULE, L>(a, max_portions, stream);
}

template <int RULE>
int launch_lanes(RuleArgs& a, int tokens, int max_portions, cudaStream_t stream) {
  int lanes = 1;                     // threads that share a column
  while (lanes * ROWS < a.dk) lanes *= 2;
  switch (lanes) {
    case 1: return launch<RULE, 1>(a, tokens, max_portions, stream);
    case 2: return launch<RULE, 2>(a, tokens, max_portions, stream);
    case 4: return launch<RULE, 4>(a, tokens, max_portions, stream);
    case 8: return launch<RULE, 8>(a, tokens, max_portions, stream);
    case 16: return launch<RULE, 16>(a, tokens, max_portions, stream);
    case 32: return launch<RULE, 32>(a, tokens, max_portions, stream);
  }
  return LS_E_SIZE;
}

}  // namespace
