// Tensor-core forms of attention with mixed heads: not built yet, every shape takes the plain kernel (seq_attn.cu).
#include "seq_attn_mma.cuh"

namespace wf {
namespace seq {

bool talk_attn_mma_usable(const GqaDims&, const PagedCache&) { return false; }
size_t talk_attn_workspace(const GqaDims&, int, int) { return 0; }
int launch_talk_attn_mma(const Batch&, const GqaDims&, const void*, const PagedCache&, void*, float*, int, cudaStream_t) {
    set_error("attention: no tensor-core form with mixed heads");
    return WF_ERR_UNSUPPORTED;
}

}  // namespace seq
}  // namespace wf
