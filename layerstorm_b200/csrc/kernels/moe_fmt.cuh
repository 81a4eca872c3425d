// Byte layout of one expert slot in the expert arena, shared by the weight-streaming MoE kernels
// (moe.cu) and the tensor-core grouped GEMM (moe_tc.cu).  Mirrors the ctypes structure of the same
// name on the Python side.
#pragma once

namespace lsb {

struct ExpertFmt {
    int fmt;                 // gate / up: 0 bf16, 1 fp8 block-128, 2 nvfp4, 3 GGUF Q4_K, 4 Q5_K, 5 Q6_K (224-byte blocks), 6 Q8_0 (planar rows), 7 fp32 (fp32 activations)
    int H, F;                // hidden, expert intermediate
    long long stride;        // bytes between slots
    long long off_gate, off_up, off_down;        // weights
    long long off_sg, off_su, off_sd;            // scales (fp8: fp32 block scales; nvfp4: atoms)
    long long off_tail;                           // nvfp4: 3 fp32 per-tensor scales (gate, up, down)
    int fmt_down1;                                // format of the down matrix + 1 when it differs from `fmt` (GGUF files mix block
                                                  // types per tensor), 0 = same as `fmt`
    __host__ __device__ int down_fmt() const { return fmt_down1 ? fmt_down1 - 1 : fmt; }
};

// Activation of a gated unit: g = min(g, limit), u = clamp(u, -limit, limit) (limit 0: as they are), then g sigmoid(alpha g) (u + shift).
// in_scale: one factor per (row, slot) pair on the unit's input - the products are linear in it, so it multiplies g and u in fp32 - or null.
// unit 1: no gate, the square of relu(u).
struct GluAct { float limit, alpha, shift; const float* in_scale; int unit = 0; };

#ifdef __CUDACC__
__device__ __forceinline__ float relu2_act(float u) { const float r = fmaxf(u, 0.f); return r * r; }
template <bool EXACT = false> __device__ __forceinline__ float glu_act(float g, float u, const GluAct& a) {
    if (a.limit > 0.f) { g = fminf(g, a.limit); u = fminf(fmaxf(u, -a.limit), a.limit); }
    if (EXACT) return g / (1.f + expf(-a.alpha * g)) * (u + a.shift);
    return __fdividef(g, 1.f + __expf(-a.alpha * g)) * (u + a.shift);
}
__device__ __forceinline__ float glu_in_scale(const GluAct& a, int pair) { return a.in_scale ? a.in_scale[pair] : 1.f; }
#endif

}  // namespace lsb
