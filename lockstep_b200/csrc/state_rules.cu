// The launcher of the state rules (state_rules.cuh), and the instances of the rules without a delta.
#include "state_rules.cuh"

int ls_launch_delta_rules(int rule, void* args, int tokens, int max_portions, cudaStream_t stream);

// `rule`: RULE_*.  `dtype`: the engine's type (of carry_src, and of r or q, k and v where they are not float32 rows).
// `tokens`: the step's tokens (`max_portions` of them or fewer: every portion may be a single token).
LS_API int ls_state_rule(int rule, int dtype, const int* portions, int max_portions, int tokens, float* state,
                         int64_t state_stride, const void* in_a, const void* in_b, const void* in_v, const float* decay,
                         const float* beta, const float* bonus, float* out, const void* carry_src, int64_t carry_ld,
                         int carry_width, int carry_rows, int H, int G, int dk, int dv, int64_t in_ld, float out_scale,
                         int64_t decay_ld, const float* gate_bias, float gate_cap, cudaStream_t stream) {
  if (max_portions <= 0 || tokens <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > 32 * ROWS || dv <= 0 || carry_rows < 0 || carry_rows >= MAX_TAPS) return LS_E_SIZE;
  if (H > 65535) return LS_E_SIZE;
  if (dtype != LS_F32 && dtype != LS_BF16) return LS_E_DTYPE;
  RuleArgs a;
  a.portions = portions; a.state = state; a.state_stride = state_stride; a.in_a = in_a; a.in_b = in_b; a.in_v = in_v;
  a.decay = decay; a.beta = beta; a.bonus = bonus; a.out = out; a.carry_src = carry_src; a.carry_ld = carry_ld;
  a.carry_width = carry_width; a.carry_rows = carry_rows; a.H = H; a.G = G; a.dk = dk; a.dv = dv;
  a.bf16 = dtype == LS_BF16 ? 1 : 0;
  a.walkers = 0;
  a.in_ld = in_ld; a.out_scale = out_scale;
  a.decay_ld = decay_ld < 0 ? (int64_t)H * dk : decay_ld;
  a.gate_bias = gate_bias; a.gate_cap = gate_cap;
  {
    const bool delta = rule == RULE_DELTA || rule == RULE_DELTA_HEAD, columns = rule == RULE_GLA || rule == RULE_MLSTM;
    const int size = delta || !a.bf16 ? 4 : 2;
    const int64_t row = delta ? 2 * (int64_t)G * dk + (int64_t)H * dv : columns ? in_ld : (int64_t)H * dk;
    auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
    a.pieces = (dk * size) % 16 == 0 && (row * size) % 16 == 0 && aligned(in_a) && (delta || aligned(in_b)) &&
               (delta || (reinterpret_cast<uintptr_t>(in_v) & 3) == 0) && (rule != RULE_WKV || (H * dv * size) % 4 == 0) &&
               (rule == RULE_DELTA_HEAD || rule == RULE_MLSTM || (dk % 4 == 0 && aligned(decay)));
  }
  switch (rule) {
    case RULE_DELTA:
      LS_COUNT(LS_K_DELTA_RULE);
      return ls_launch_delta_rules(rule, &a, tokens, max_portions, stream);
    case RULE_WKV:
      LS_COUNT(LS_K_WKV_RULE);
      return launch_lanes<RULE_WKV>(a, tokens, max_portions, stream);
    case RULE_GLA:
      if (H != G || in_ld <= 0) return LS_E_SIZE;
      LS_COUNT(LS_K_GLA_RULE);
      return launch_lanes<RULE_GLA>(a, tokens, max_portions, stream);
    case RULE_DELTA_HEAD:
      LS_COUNT(LS_K_DELTA_HEAD_RULE);
      return ls_launch_delta_rules(rule, &a, tokens, max_portions, stream);
    case RULE_MLSTM:
      if (H != G || in_ld <= 0 || gate_bias == nullptr || !(gate_cap > 0.f) || carry_rows != 0) return LS_E_SIZE;
      LS_COUNT(LS_K_MLSTM_RULE);
      return launch_lanes<RULE_MLSTM>(a, tokens, max_portions, stream);
  }
  return LS_E_SIZE;
}

LS_API const char* ls_constants_state_rules() {
  static char buf[256];
  static const LsConstant c[] = {{"state_rules.rows_per_thread", ROWS}, {"state_rules.chunk_tokens", CHUNK},
                                 {"state_rules.staging_threads", STAGERS}};
  return ls_format_constants(buf, sizeof buf, c, (int)(sizeof c / sizeof c[0]));
}
