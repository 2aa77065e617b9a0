// Prompt attention over key and value pages without a distance bias: instances of the window attention kernel, compiled
// apart from those with one (grouped_attn.cu).
#include "attn_window.cuh"

namespace bcg {

int window_attn_paged(int q_ld, int v_ld, const CUtensorMap& qm, const CUtensorMap& km, const CUtensorMap& vm,
                      const WindowAttn& a, cudaStream_t st) {
  return window_attn<true, false>(q_ld, v_ld, qm, km, vm, a, st);
}

}  // namespace bcg
