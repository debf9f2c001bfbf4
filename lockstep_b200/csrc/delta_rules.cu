// The instances of the gated delta rule (state_rules.cuh), in a source of their own so that they compile beside the others.
#include "state_rules.cuh"

int ls_launch_delta_rules(int rule, void* args, int tokens, int max_portions, cudaStream_t stream) {
  RuleArgs& a = *reinterpret_cast<RuleArgs*>(args);
  if (rule == RULE_DELTA) return launch_lanes<RULE_DELTA>(a, tokens, max_portions, stream);
  return launch_lanes<RULE_DELTA_HEAD>(a, tokens, max_portions, stream);
}
