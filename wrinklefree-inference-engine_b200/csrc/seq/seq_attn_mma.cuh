// Pieces shared by the tensor-core attention kernels: ldmatrix / mma.sync / cp.async wrappers, the softmax denominator with a sink.
#pragma once
#include "seq_kernels.cuh"

namespace wf {
namespace seq {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void am_ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void am_ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void am_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void am_cp16(uint32_t dst, const void* src, bool valid) {
    const int sz = valid ? 16 : 0;          // 0: the 16 bytes are zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(sz) : "memory");
}
__device__ __forceinline__ void am_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void am_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}

// 1 / (sum + the extra key's share), scaled by 2^m of the running maximum m (units of log 2): the extra key's score is 0 or a learned one,
// which may exceed every score, so both are brought to the larger maximum.  The weighted values are multiplied by the result.
__device__ __forceinline__ float am_inv_sum(const GqaDims& D, int head, float m, float l) {
    if (!D.sink) return 1.f / l;
    const float ms = D.sink_h ? D.sink_h[head] * LOG2E : 0.f, top = fmaxf(m, ms), f = exp2f(m - top);
    return f / (l * f + exp2f(ms - top));
}

}  // namespace seq
}  // namespace wf
