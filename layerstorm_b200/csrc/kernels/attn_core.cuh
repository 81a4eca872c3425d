// Pieces shared by the softmax-attention kernels over the paged cache (attn.cu: grouped heads, latent.cu: one latent row for all heads): the
// parameter block, the CUDA-core kernel, and the mma.sync / cp.async helpers.
#pragma once
#include "common.cuh"

namespace lsb {

struct AttnParams {
    const void* q;                    // [rows, H, dkp] bf16 / fp32
    const void* cache; const int* block_table; int max_pages, page;
    const int* row_seq; const int* row_pos;
    const float* proj; int ldp, off_gate, head_gate;     // gate per value channel, or (head_gate) one per head
    int ldc, off_v;                   // cache row: elements, and where the values start (latent rows: 0, the values are the head of the key row)
    int dkh, off_ks;                  // key channels from dkh on are shared by all heads and start at element off_ks of the row (dkh = dkp: none)
    void* out; int ldo;               // [rows, ldo]
    float* o_part; float* ml_part;    // [rows, H, NS, dvp], [rows, H, NS, 2]
    int rows, H, G, dk, dv, dkp, dvp, NS, window;
    float scale;
    const float* slope;               // [H] (log2 units are applied in the kernels) or null
    int chunk = 0;                    // a position sees the keys of its own chunk of this many (0: no chunks)
    const float* bias = nullptr;      // [H, bias_len] added to the scores by distance, the last entry for all further ones; or null
    int bias_len = 0;
    float out_scale = 1.f;            // on the heads' outputs
    int maps = 1;                     // consecutive groups that attend over one value head (G / maps value heads)
    const float* sink = nullptr;      // [H] a term exp(sink) that only the softmax's denominator has, or null
    float* out32 = nullptr;           // [rows, H, dvp] fp32 results in place of `out`, without gate and factor
    int key_base = 0;                 // position of the cache's first row (caches that are one page)
};

// first key that position `pos` sees
__device__ __forceinline__ int attn_low(const AttnParams& p, int pos) {
    const int w = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    return p.chunk > 0 ? max(w, pos / p.chunk * p.chunk) : w;
}

template <typename T> __device__ __forceinline__ T to_act(float v);
template <> __device__ __forceinline__ bf16 to_act<bf16>(float v) { return __float2bfloat16(v); }
template <> __device__ __forceinline__ float to_act<float>(float v) { return v; }
__device__ __forceinline__ float act_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float act_f(float v) { return v; }
__device__ __forceinline__ float gate_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
// factor on value channel c of head h: output gate (if any) and constant
__device__ __forceinline__ float attn_out_factor(const AttnParams& p, size_t r, int h, int c) {
    return p.off_gate >= 0 ? p.out_scale * gate_sigmoid(p.proj[r * p.ldp + p.off_gate + (p.head_gate ? (size_t)h : (size_t)h * p.dv + c)]) : p.out_scale;
}

// 1 / denominator, relative to the running maximum m (log2 units; never -inf) of head h's scores with sum l
__device__ __forceinline__ float attn_inv_sum(const AttnParams& p, int h, float m, float l) {
    if (!p.sink) return 1.f / l;
    const float s = p.sink[h] * 1.4426950408889634f, M = fmaxf(m, s), f = exp2f(m - M);
    return f / fmaf(l, f, exp2f(s - M));
}

// cosine and sine of pos * freq; the angle is reduced in fp64 so that far positions keep their phase
__device__ __forceinline__ void rotary_angle(int pos, double freq, float& s, float& c) {
    constexpr double kTwoPi = 6.283185307179586476925;
    const double x = (double)pos * freq;
    sincosf((float)(x - kTwoPi * rint(x * (1.0 / kTwoPi))), &s, &c);
}

// ------------------------------------------------------------------------------------------------ CUDA-core kernel
// One block per (row, head): 128 keys at a time, one thread per key for the scores, one per value channel for the sum.
template <typename T>
static __global__ void __launch_bounds__(128) attn_exact_kernel(AttnParams p) {
    extern __shared__ __align__(16) float esm[];
    float* s_q = esm;                                     // [dkp]
    float* s_p = s_q + p.dkp;                             // [128]
    int* s_row = reinterpret_cast<int*>(s_p + 128);       // [128] cache row of the tile's keys
    float* s_o = reinterpret_cast<float*>(s_row + 128);   // [dv]
    __shared__ float red[33];
    const int r = blockIdx.x, h = blockIdx.y, t = threadIdx.x, g = h / (p.H / p.G);
    pdl_wait();
    pdl_launch_dependents();
    const int seq = p.row_seq[r], pos = p.row_pos[r];
    if (seq < 0) return;
    const T* q = reinterpret_cast<const T*>(p.q) + ((size_t)r * p.H + h) * p.dkp;
    for (int i = t; i < p.dkp; i += 128) s_q[i] = act_f(q[i]);
    for (int i = t; i < p.dv; i += 128) s_o[i] = 0.f;
    const float slope = p.slope ? p.slope[h] : 0.f;
    const size_t ldc = (size_t)p.ldc;
    const T* cache = reinterpret_cast<const T*>(p.cache);
    const int lo = attn_low(p, pos);
    const float* bias = p.bias ? p.bias + (size_t)h * p.bias_len : nullptr;
    float m = -INFINITY, l = 0.f;
    for (int k0 = lo; k0 <= pos; k0 += 128) {
        const int j = k0 + t;
        float s = -INFINITY;
        int row = 0;
        __syncthreads();
        if (j <= pos) {
            row = p.block_table[(size_t)seq * p.max_pages + j / p.page] * p.page + j % p.page;
            const T* k = cache + (size_t)row * ldc + (size_t)g * p.dkp;
            float a = 0.f;
#pragma unroll 8
            for (int c = 0; c < p.dk; ++c) a = fmaf(s_q[c], act_f(k[c]), a);
            s = a * p.scale - slope * (float)(pos - j) + (bias ? bias[min(pos - j, p.bias_len - 1)] : 0.f);
        }
        s_row[t] = row;
        const float mt = fmaxf(m, block_max(s, red));
        const float e = j <= pos ? expf(s - mt) : 0.f;
        const float corr = m == -INFINITY ? 0.f : expf(m - mt);
        s_p[t] = e;
        l = l * corr + block_sum(e, red);
        m = mt;
        __syncthreads();
        const int n = min(128, pos - k0 + 1);
        for (int c = t; c < p.dv; c += 128) {
            float a = s_o[c] * corr;
            for (int i = 0; i < n; ++i) a = fmaf(s_p[i], act_f(cache[(size_t)s_row[i] * ldc + (size_t)p.off_v + (size_t)(g / p.maps) * p.dvp + c]), a);
            s_o[c] = a;
        }
    }
    const float inv = attn_inv_sum(p, h, m * 1.4426950408889634f, l);
    for (int c = t; c < p.dv; c += 128) {
        if (p.out32) { p.out32[((size_t)r * p.H + h) * p.dvp + c] = s_o[c] * inv; continue; }
        const float o = s_o[c] * inv * attn_out_factor(p, r, h, c);
        reinterpret_cast<T*>(p.out)[(size_t)r * p.ldo + (size_t)h * p.dv + c] = to_act<T>(o);
    }
}

// ------------------------------------------------------------------------------------------------ tensor-core pieces (mma.sync m16n8k16)
__device__ __forceinline__ uint32_t sm_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(sm_addr(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(sm_addr(p)));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp16(bf16* dst, const bf16* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(sm_addr(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// two weights -> packed bf16 (hi) and the packed remainders (lo)
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    const bf162 h = __floats2bfloat162_rn(a, b);
    const bf162 r = __floats2bfloat162_rn(a - __low2float(h), b - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&r);
}
constexpr float kLog2e = 1.4426950408889634f;

}  // namespace lsb
