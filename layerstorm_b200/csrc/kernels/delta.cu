// Gated delta rule with one decay per key channel or per head, for any head geometry: `H` value heads of `dv` channels over `G` query / key
// heads of `dk` channels (head h reads query / key head h / (H / G)), short causal convolutions of any length, low-rank decay and output gates.
// Rank 0 of the decay: one decay per head, x = its column of the projection.  Rank 0 of the output gate: SiLU of a full-rank projection.
//
//   q, k, v = SiLU(conv(raw));  q = q / sqrt(sum q^2 + 1e-6) * q_scale;  k = k / sqrt(sum k^2 + 1e-6)
//   log g = decay(a_exp[h], W_a a + dt_bias)      one per head and key channel; mode 0: -a_exp softplus(x), mode 1: bound * sigmoid(a_exp x)
//   S <- g * S;  u = sigmoid(b) (v - S^T k);  S <- S + k u^T;  o = S^T q          (decay, read, write, read out)
//   out = o / sqrt(mean(o^2) + eps) * w_onorm * sigmoid(W_g g1)
//
// State: fp32 [slots, H, dv, DKP], one row of DKP (dk padded to 32 / 64 / 128 / 256) floats per value channel; convolution history: fp32
// [slots, H, 2 dk + dv, taps - 1], oldest first - every head keeps its own copy of its query / key channels, so a block never reads what
// another block of the same launch writes.  The key channels of a value channel are spread over four lanes.  Both reductions of a token
// run over the decayed state (S^T k and S^T q), because S_new^T q = (g S)^T q + u (k . q).
//
// Few rows per sequence: one kernel (delta_step).  Longer runs: delta_prep (everything outside the recurrence, parallel over rows), the
// recurrence (chunk-parallel for long sequences, see kda_chunk.cuh; token by token otherwise), delta_out.
#include <cstdlib>
#include "common.cuh"

namespace lsb {

#include "kda_types.cuh"
#include "kda_chunk.cuh"

struct DeltaParams {
    const float* proj;                      // [rows, ldp] fp32: q | k | v | b | a | g at the offsets below
    int ldp, off_q, off_k, off_v, off_b, off_a, off_g;
    int rank_a, rank_g;                     // padded to multiples of 8
    const void* w_a;                        // [H * dk, rank_a]
    const void* w_g;                        // [H * dv, rank_g]
    const float* conv_q; const float* conv_k; const float* conv_v;      // [G dk | G dk | H dv, taps], last column = the current token
    const float* a_exp; const float* dt_bias; const float* onorm;       // [H], [H * dk], [dv]
    float* state; float* conv_state;
    const int* seq_row0; const int* seq_nrows; const int* seq_slot;
    void* out; int ldo;                     // [rows, ldo], bf16 or fp32
    int H, G, dk, dv, taps, decay_mode;
    float q_scale, decay_bound, eps;
};

struct DeltaScratch {
    float* qn; float* kn; float* ld;        // [rows, H, DKP]: unit vectors (q scaled), log decay
    float* vo;                              // [rows, H, dv]   v in, o out
    float* beta; float* kq;                 // [rows, H]       k . q of the unit vectors
    float* rawa; float* rawg;               // [rows, H dk], [rows, H dv]  low-rank products
};

__device__ __forceinline__ float sigmoid_acc(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float delta_log_decay(int mode, float a_exp, float x, float bound) {
    if (mode == 0) return -a_exp * (x > 20.f ? x : log1pf(expf(x)));
    return bound * sigmoid_acc(a_exp * x);
}

// rank_a 0: the head's log decay at a row of the projection;  rank_g 0: the output gate of value channel v
__device__ __forceinline__ float delta_head_decay(const DeltaParams& p, const float* pr, int h, float a_exp) {
    return delta_log_decay(p.decay_mode, a_exp, pr[p.off_a + h] + p.dt_bias[h], p.decay_bound);
}
__device__ __forceinline__ float delta_full_gate(const DeltaParams& p, const float* pr, int h, int v) {
    const float x = pr[p.off_g + (size_t)h * p.dv + v];
    return x * sigmoid_acc(x);
}

// channel c of a head: [0, dk) query, [dk, 2 dk) key, [2 dk, 2 dk + dv) value -> projection column and convolution taps
__device__ __forceinline__ void delta_channel(const DeltaParams& p, int h, int c, int& col, const float*& w) {
    const int gh = h / (p.H / p.G);
    if (c < p.dk) { const int ch = gh * p.dk + c; col = p.off_q + ch; w = p.conv_q + (size_t)ch * p.taps; }
    else if (c < 2 * p.dk) { const int ch = gh * p.dk + c - p.dk; col = p.off_k + ch; w = p.conv_k + (size_t)ch * p.taps; }
    else { const int ch = h * p.dv + c - 2 * p.dk; col = p.off_v + ch; w = p.conv_v + (size_t)ch * p.taps; }
}
__device__ __forceinline__ float* delta_history(const DeltaParams& p, int slot, int h, int c) {
    return p.conv_state + (((size_t)slot * p.H + h) * (2 * p.dk + p.dv) + c) * (p.taps - 1);
}
// convolution output (after SiLU) of channel c at row i of a sequence whose step rows start at row0
__device__ __forceinline__ float delta_conv(const DeltaParams& p, int h, int c, int slot, int row0, int i) {
    int col; const float* w;
    delta_channel(p, h, c, col, w);
    const float* hist = delta_history(p, slot, h, c);
    float y = 0.f;
#pragma unroll 4
    for (int d = 0; d < p.taps; ++d) {
        const int j = i - (p.taps - 1) + d;                        // row of tap d inside the step
        const float x = j >= 0 ? p.proj[(size_t)(row0 + j) * p.ldp + col] : hist[p.taps - 1 + j];
        y = fmaf(x, w[d], y);
    }
    return y * sigmoid_acc(y);
}
// the history after `nrows` rows: the last taps - 1 raw inputs (one thread per channel; ascending order never reads what it wrote)
__device__ __forceinline__ void delta_push_history(const DeltaParams& p, int h, int c, int slot, int row0, int nrows) {
    int col; const float* w;
    delta_channel(p, h, c, col, w);
    float* hist = delta_history(p, slot, h, c);
    for (int d = 0; d < p.taps - 1; ++d) {
        const int j = nrows - (p.taps - 1) + d;
        hist[d] = j >= 0 ? p.proj[(size_t)(row0 + j) * p.ldp + col] : hist[p.taps - 1 + j];
    }
}

template <typename T> __device__ __forceinline__ void store_act(void* out, size_t i, float v);
template <> __device__ __forceinline__ void store_act<bf16>(void* out, size_t i, float v) { reinterpret_cast<bf16*>(out)[i] = __float2bfloat16(v); }
template <> __device__ __forceinline__ void store_act<float>(void* out, size_t i, float v) { reinterpret_cast<float*>(out)[i] = v; }

__device__ __forceinline__ float quad_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    return v + __shfl_xor_sync(0xffffffffu, v, 2);
}

// dot of a row of a low-rank matrix with an fp32 vector, spread over the four lanes of a quad (16-byte pieces in turn)
template <typename T> __device__ __forceinline__ float quad_dot(const uint8_t* row, const float* x, int rank, int ks);
template <> __device__ __forceinline__ float quad_dot<bf16>(const uint8_t* row, const float* x, int rank, int ks) {
    float a = 0.f;
    for (int j = ks * 8; j < rank; j += 32) {
        float f[8];
        unpack_bf16x8(*reinterpret_cast<const uint4*>(row + (size_t)j * 2), f);
#pragma unroll
        for (int e = 0; e < 8; ++e) a = fmaf(f[e], x[j + e], a);
    }
    return quad_sum(a);
}
template <> __device__ __forceinline__ float quad_dot<float>(const uint8_t* row, const float* x, int rank, int ks) {
    float a = 0.f;
    for (int j = ks * 4; j < rank; j += 16) {
        const float4 f = *reinterpret_cast<const float4*>(row + (size_t)j * 4);
        a = fmaf(f.x, x[j], a); a = fmaf(f.y, x[j + 1], a); a = fmaf(f.z, x[j + 2], a); a = fmaf(f.w, x[j + 3], a);
    }
    return quad_sum(a);
}

// Shared-memory row stride of a staged low-rank matrix: the quads of a quarter warp start 64 bytes apart modulo 128.
__host__ __device__ constexpr int delta_gate_row_bytes(int rank_bytes) { return (rank_bytes + 127) / 128 * 128 + 64; }

// ------------------------------------------------------------------------------------------------ few rows
// One block per (sequence, head), four threads per value channel.  `staged`: the head's low-rank rows come through shared memory.
template <int DKP, int MAXT, typename WT, typename OT>
__global__ void __launch_bounds__(MAXT, 1) delta_step_kernel(DeltaParams p, int staged) {
    constexpr int NJ = DKP / 16;                                   // 16-byte pieces of the key channels per lane
    extern __shared__ __align__(16) uint8_t dsm[];
    const int T = blockDim.x, t = threadIdx.x, lane = t & 31, ks = t & 3;
    const int seq = blockIdx.x, h = blockIdx.y;
    float* s_x = reinterpret_cast<float*>(dsm);                    // [2 DKP] q | k after convolution
    float* s_g = s_x + 2 * DKP;                                    // [DKP] decay factors
    float* s_v = s_g + DKP;                                        // [dv]
    float* s_fa = s_v + p.dv;                                      // [rank_a]
    float* s_ga = s_fa + p.rank_a;                                 // [rank_g]
    float* s_red = s_ga + p.rank_g;                                // [33]
    uint8_t* s_w = dsm + (((size_t)(3 * DKP + p.dv + p.rank_a + p.rank_g + 33) * 4 + 15) & ~(size_t)15);
    const int row0 = p.seq_row0[seq], nrows = p.seq_nrows[seq], slot = p.seq_slot[seq];
    const int rba = p.rank_a * (int)sizeof(WT), rbg = p.rank_g * (int)sizeof(WT);
    const int sra = staged ? delta_gate_row_bytes(rba) : rba, srg = staged ? delta_gate_row_bytes(rbg) : rbg;
    const uint8_t* ga_src = reinterpret_cast<const uint8_t*>(p.w_a) + (size_t)h * p.dk * rba;
    const uint8_t* gg_src = reinterpret_cast<const uint8_t*>(p.w_g) + (size_t)h * p.dv * rbg;
    const uint8_t* wa = ga_src;
    const uint8_t* wg = gg_src;
    if (staged) {
        uint8_t* da = s_w;
        uint8_t* dg = s_w + (size_t)p.dk * sra;
        for (int i = t; i < p.dk * (rba / 16); i += T) {
            const int r = i / (rba / 16), c = i - r * (rba / 16);
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(da + (size_t)r * sra + c * 16)), "l"(ga_src + (size_t)i * 16) : "memory");
        }
        for (int i = t; i < p.dv * (rbg / 16); i += T) {
            const int r = i / (rbg / 16), c = i - r * (rbg / 16);
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dg + (size_t)r * srg + c * 16)), "l"(gg_src + (size_t)i * 16) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        wa = da; wg = dg;
    }
    const bool live = nrows > 0 && slot >= 0;
    const int v = t >> 2;
    const bool has_v = v < p.dv;
    float4 S[NJ];
    float* sp = p.state + (((size_t)(live ? slot : 0) * p.H + h) * p.dv + (has_v ? v : 0)) * DKP + ks * 4;
    if (live && has_v) {
#pragma unroll
        for (int j = 0; j < NJ; ++j) S[j] = *reinterpret_cast<const float4*>(sp + j * 16);
    } else {
#pragma unroll
        for (int j = 0; j < NJ; ++j) S[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int c = t; c < 3 * DKP; c += T) s_x[c] = 0.f;              // padding channels: no key, no query, an empty state column
    pdl_wait();
    pdl_launch_dependents();
    if (!live) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        return;
    }
    const float a_exp = p.a_exp[h];
    const float ow = has_v ? p.onorm[v] : 0.f;
    const int nch = 2 * p.dk + p.dv;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    for (int i = 0; i < nrows; ++i) {
        const float* pr = p.proj + (size_t)(row0 + i) * p.ldp;
        for (int c = t; c < nch; c += T) {
            const float y = delta_conv(p, h, c, slot, row0, i);
            if (c < 2 * p.dk) s_x[c < p.dk ? c : DKP + c - p.dk] = y; else s_v[c - 2 * p.dk] = y;
        }
        for (int c = t; c < p.rank_a + p.rank_g; c += T) s_fa[c] = c < p.rank_a ? pr[p.off_a + c] : pr[p.off_g + c - p.rank_a];
        const float beta = sigmoid_acc(pr[p.off_b + h]);
        __syncthreads();
        // every warp takes the three sums over the key channels on its own
        float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
        for (int c = 0; c < DKP / 32; ++c) {
            const float a = s_x[lane + 32 * c], b = s_x[DKP + lane + 32 * c];
            qq = fmaf(a, a, qq); kk = fmaf(b, b, kk); qk = fmaf(a, b, qk);
        }
        qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
        const float qi = p.q_scale / sqrtf(qq + 1e-6f), ki = 1.f / sqrtf(kk + 1e-6f);
        float gate = 0.f;
        if (p.rank_g == 0) gate = delta_full_gate(p, pr, h, has_v ? v : 0);
        else if (p.dv == (T >> 2) || __any_sync(0xffffffffu, has_v))
            gate = sigmoid_acc(quad_dot<WT>(wg + (size_t)(has_v ? v : 0) * srg, s_ga, p.rank_g, ks));
        if (p.rank_a == 0) {
            const float gh = expf(delta_head_decay(p, pr, h, a_exp));
            for (int c = t; c < p.dk; c += T) s_g[c] = gh;
        } else for (int c0 = 0; c0 < p.dk; c0 += T >> 2) {
            const int c = c0 + v;
            const float x = quad_dot<WT>(wa + (size_t)min(c, p.dk - 1) * sra, s_fa, p.rank_a, ks);
            if (ks == 0 && c < p.dk) s_g[c] = expf(delta_log_decay(p.decay_mode, a_exp, x + p.dt_bias[(size_t)h * p.dk + c], p.decay_bound));
        }
        __syncthreads();
        const float4* q4 = reinterpret_cast<const float4*>(s_x) + ks;
        const float4* k4 = reinterpret_cast<const float4*>(s_x + DKP) + ks;
        const float4* g4 = reinterpret_cast<const float4*>(s_g) + ks;
        float4 sk = make_float4(0.f, 0.f, 0.f, 0.f), sq = sk;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const float4 g = g4[j * 4], k = k4[j * 4], q = q4[j * 4];
            S[j].x *= g.x; S[j].y *= g.y; S[j].z *= g.z; S[j].w *= g.w;
            sk.x = fmaf(S[j].x, k.x, sk.x); sk.y = fmaf(S[j].y, k.y, sk.y); sk.z = fmaf(S[j].z, k.z, sk.z); sk.w = fmaf(S[j].w, k.w, sk.w);
            sq.x = fmaf(S[j].x, q.x, sq.x); sq.y = fmaf(S[j].y, q.y, sq.y); sq.z = fmaf(S[j].z, q.z, sq.z); sq.w = fmaf(S[j].w, q.w, sq.w);
        }
        const float skt = quad_sum((sk.x + sk.y) + (sk.z + sk.w)) * ki;
        const float sqt = quad_sum((sq.x + sq.y) + (sq.z + sq.w)) * qi;
        const float u = beta * ((has_v ? s_v[v] : 0.f) - skt);
        const float o = has_v ? fmaf(u, qk * qi * ki, sqt) : 0.f;
        const float uk = u * ki;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const float4 k = k4[j * 4];
            S[j].x = fmaf(uk, k.x, S[j].x); S[j].y = fmaf(uk, k.y, S[j].y); S[j].z = fmaf(uk, k.z, S[j].z); S[j].w = fmaf(uk, k.w, S[j].w);
        }
        const float os = block_sum(ks == 0 ? o * o : 0.f, s_red);
        if (ks == 0 && has_v) store_act<OT>(p.out, (size_t)(row0 + i) * p.ldo + (size_t)h * p.dv + v, o / sqrtf(os / (float)p.dv + p.eps) * ow * gate);
        __syncthreads();
    }
    if (has_v) {
#pragma unroll
        for (int j = 0; j < NJ; ++j) *reinterpret_cast<float4*>(sp + j * 16) = S[j];
    }
    for (int c = t; c < nch; c += T) delta_push_history(p, h, c, slot, row0, nrows);
}

// ------------------------------------------------------------------------------------------------ many rows
// fp32 low-rank activations -> bf16 (hi | lo) pairs: with the duplicated weights [W | W] the bf16 tensor-core product then equals the
// product with fp32 activations to ~2^-16.  xs[row] = [a_hi | a_lo | g_hi | g_lo].
__global__ void __launch_bounds__(128) delta_split_kernel(const float* __restrict__ proj, int ldp, int off_a, int rank_a, int off_g, int rank_g,
                                                          bf16* __restrict__ xs) {
    pdl_wait();
    pdl_launch_dependents();
    const int row = blockIdx.x, ra2 = 2 * rank_a, ld = ra2 + 2 * rank_g;
    const float* pr = proj + (size_t)row * ldp;
    bf16* o = xs + (size_t)row * ld;
    for (int j = threadIdx.x; j < rank_a + rank_g; j += blockDim.x) {
        const bool a = j < rank_a;
        const float v = a ? pr[off_a + j] : pr[off_g + j - rank_a];
        const bf16 hi = __float2bfloat16(v);
        const int d = a ? j : ra2 + j - rank_a;
        o[d] = hi;
        o[d + (a ? rank_a : rank_g)] = __float2bfloat16(v - __bfloat162float(hi));
    }
}

constexpr int kDeltaPrepRows = 16;

// One warp per (row, head): convolutions, unit vectors, log decays, write strength.
template <int DKP>
__global__ void __launch_bounds__(128) delta_prep_kernel(DeltaParams p, DeltaScratch w, int nseq, int total_rows) {
    constexpr int NC = DKP / 32;
    const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_wait();
    pdl_launch_dependents();
    const float a_exp = p.a_exp[h];
    const int row_end = min(total_rows, (int)(blockIdx.x + 1) * kDeltaPrepRows);
    for (int row = blockIdx.x * kDeltaPrepRows + warp; row < row_end; row += 4) {
        int row0 = -1, slot = 0;
        for (int s = 0; s < nseq; ++s) {
            const int r0 = p.seq_row0[s], n = p.seq_nrows[s];
            if (row >= r0 && row < r0 + n) { row0 = r0; slot = p.seq_slot[s]; break; }
        }
        if (row0 < 0) continue;                                    // no sequence of this step (warp-uniform)
        const int i = row - row0;
        float q[NC], k[NC], qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
        for (int j = 0; j < NC; ++j) {
            const int c = lane + 32 * j;
            q[j] = c < p.dk ? delta_conv(p, h, c, slot, row0, i) : 0.f;
            k[j] = c < p.dk ? delta_conv(p, h, p.dk + c, slot, row0, i) : 0.f;
            qq = fmaf(q[j], q[j], qq); kk = fmaf(k[j], k[j], kk); qk = fmaf(q[j], k[j], qk);
        }
        qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
        const float qi = p.q_scale / sqrtf(qq + 1e-6f), ki = 1.f / sqrtf(kk + 1e-6f);
        const size_t o = ((size_t)row * p.H + h) * DKP;
#pragma unroll
        for (int j = 0; j < NC; ++j) {
            const int c = lane + 32 * j;
            w.qn[o + c] = q[j] * qi;
            w.kn[o + c] = k[j] * ki;
            if (p.rank_a == 0) w.ld[o + c] = c < p.dk ? delta_head_decay(p, p.proj + (size_t)row * p.ldp, h, a_exp) : 0.f;
            else w.ld[o + c] = c < p.dk ? delta_log_decay(p.decay_mode, a_exp, w.rawa[((size_t)row * p.H + h) * p.dk + c] + p.dt_bias[(size_t)h * p.dk + c], p.decay_bound) : 0.f;
        }
        for (int c = lane; c < p.dv; c += 32) w.vo[((size_t)row * p.H + h) * p.dv + c] = delta_conv(p, h, 2 * p.dk + c, slot, row0, i);
        if (lane == 0) {
            w.beta[(size_t)row * p.H + h] = sigmoid_acc(p.proj[(size_t)row * p.ldp + p.off_b + h]);
            w.kq[(size_t)row * p.H + h] = qk * qi * ki;
        }
    }
}

// The recurrence token by token: one block per (sequence, head, 32 value channels), key vectors through a double-buffered cp.async ring.
// Sequences of `max_rows` rows or more are left to the chunk kernels.
template <int DKP>
__global__ void __launch_bounds__(128) delta_recur_kernel(DeltaParams p, DeltaScratch w, int max_rows) {
    constexpr int NJ = DKP / 16, TCH = DKP > 128 ? 4 : 8, PCS = DKP / 4;
    __shared__ __align__(16) float sm[2][3][TCH][DKP];             // [buffer][q, k, log decay -> decay][token][channel]
    const int seq = blockIdx.x, h = blockIdx.y, t = threadIdx.x, ks = t & 3, v = blockIdx.z * 32 + (t >> 2);
    pdl_wait();
    pdl_launch_dependents();
    const int row0 = p.seq_row0[seq], nrows = p.seq_nrows[seq], slot = p.seq_slot[seq];
    if (nrows <= 0 || slot < 0 || nrows >= max_rows) return;
    const bool has_v = v < p.dv;
    float4 S[NJ];
    float* sp = p.state + (((size_t)slot * p.H + h) * p.dv + (has_v ? v : 0)) * DKP + ks * 4;
#pragma unroll
    for (int j = 0; j < NJ; ++j) S[j] = has_v ? *reinterpret_cast<const float4*>(sp + j * 16) : make_float4(0.f, 0.f, 0.f, 0.f);
    const int nchunks = (nrows + TCH - 1) / TCH;
    auto issue = [&](int chunk, int buf) {
        for (int idx = t; idx < 3 * TCH * PCS; idx += 128) {
            const int arr = idx / (TCH * PCS), rem = idx % (TCH * PCS), tok = rem / PCS, c4 = rem % PCS;
            const int row = row0 + min(chunk * TCH + tok, nrows - 1);       // rows past the end are clamped (unused)
            const float* src = (arr == 0 ? w.qn : (arr == 1 ? w.kn : w.ld)) + ((size_t)row * p.H + h) * DKP + c4 * 4;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(&sm[buf][arr][tok][c4 * 4])), "l"(src) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    issue(0, 0);
    for (int chunk = 0; chunk < nchunks; ++chunk) {
        const int buf = chunk & 1;
        if (chunk + 1 < nchunks) issue(chunk + 1, buf ^ 1); else asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        for (int idx = t; idx < TCH * DKP; idx += 128) { float* d = &sm[buf][2][0][0] + idx; *d = expf(*d); }
        __syncthreads();
        const int ntok = min(TCH, nrows - chunk * TCH);
        for (int j0 = 0; j0 < ntok; ++j0) {
            const size_t rh = (size_t)(row0 + chunk * TCH + j0) * p.H + h;
            const float vj = has_v ? w.vo[rh * p.dv + v] : 0.f, beta = w.beta[rh], kq = w.kq[rh];
            const float4* q4 = reinterpret_cast<const float4*>(sm[buf][0][j0]) + ks;
            const float4* k4 = reinterpret_cast<const float4*>(sm[buf][1][j0]) + ks;
            const float4* g4 = reinterpret_cast<const float4*>(sm[buf][2][j0]) + ks;
            float4 sk = make_float4(0.f, 0.f, 0.f, 0.f), sq = sk;
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const float4 g = g4[j * 4], k = k4[j * 4], q = q4[j * 4];
                S[j].x *= g.x; S[j].y *= g.y; S[j].z *= g.z; S[j].w *= g.w;
                sk.x = fmaf(S[j].x, k.x, sk.x); sk.y = fmaf(S[j].y, k.y, sk.y); sk.z = fmaf(S[j].z, k.z, sk.z); sk.w = fmaf(S[j].w, k.w, sk.w);
                sq.x = fmaf(S[j].x, q.x, sq.x); sq.y = fmaf(S[j].y, q.y, sq.y); sq.z = fmaf(S[j].z, q.z, sq.z); sq.w = fmaf(S[j].w, q.w, sq.w);
            }
            const float skt = quad_sum((sk.x + sk.y) + (sk.z + sk.w)), sqt = quad_sum((sq.x + sq.y) + (sq.z + sq.w));
            const float u = beta * (vj - skt);
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
                const float4 k = k4[j * 4];
                S[j].x = fmaf(u, k.x, S[j].x); S[j].y = fmaf(u, k.y, S[j].y); S[j].z = fmaf(u, k.z, S[j].z); S[j].w = fmaf(u, k.w, S[j].w);
            }
            if (ks == 0 && has_v) w.vo[rh * p.dv + v] = fmaf(u, kq, sqt);
        }
        __syncthreads();                                           // everyone is done with `buf` before it is refilled
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (has_v) {
#pragma unroll
        for (int j = 0; j < NJ; ++j) *reinterpret_cast<float4*>(sp + j * 16) = S[j];
    }
    if (blockIdx.z == 0)
        for (int c = t; c < 2 * p.dk + p.dv; c += 128) delta_push_history(p, h, c, slot, row0, nrows);
}

struct DeltaTail {
    DeltaParams p;
    __device__ void operator()(int h, int vs, int tid, int row0, int nrows, int slot) const {
        if (vs == 0)
            for (int c = tid; c < 2 * p.dk + p.dv; c += 256) delta_push_history(p, h, c, slot, row0, nrows);
    }
};

// gated RMSNorm of the outputs: one warp per (row, head)
template <typename OT>
__global__ void __launch_bounds__(128) delta_out_kernel(DeltaParams p, DeltaScratch w, int total_rows) {
    const int lane = threadIdx.x & 31;
    pdl_wait();
    pdl_launch_dependents();
    const long long rh = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (rh >= (long long)total_rows * p.H) return;
    const int row = (int)(rh / p.H), h = (int)(rh % p.H);
    const float* o = w.vo + (size_t)rh * p.dv;
    float ss = 0.f;
    for (int c = lane; c < p.dv; c += 32) ss = fmaf(o[c], o[c], ss);
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
    for (int c = lane; c < p.dv; c += 32) {
        const float gate = p.rank_g == 0 ? delta_full_gate(p, p.proj + (size_t)row * p.ldp, h, c) : sigmoid_acc(w.rawg[(size_t)rh * p.dv + c]);
        store_act<OT>(p.out, (size_t)row * p.ldo + (size_t)h * p.dv + c, o[c] * r * p.onorm[c] * gate);
    }
}

static int delta_pad(int dk) { return dk <= 32 ? 32 : (dk <= 64 ? 64 : (dk <= 128 ? 128 : 256)); }

// Value channels the one-kernel form takes: four threads each, and registers for the state rows.
static int delta_step_max_dv(int DKP) { return DKP <= 64 ? 256 : 128; }

template <int DKP, int MAXT, typename WT, typename OT>
static int launch_delta_step_t(const DeltaParams& p, int nseq, cudaStream_t st) {
    const size_t base = ((size_t)(3 * DKP + p.dv + p.rank_a + p.rank_g + 33) * 4 + 15) & ~(size_t)15;
    const size_t gates = (size_t)p.dk * delta_gate_row_bytes(p.rank_a * (int)sizeof(WT)) + (size_t)p.dv * delta_gate_row_bytes(p.rank_g * (int)sizeof(WT));
    const int staged = base + gates <= 200 * 1024;
    static bool attr = false;
    if (!attr) { cudaFuncSetAttribute(delta_step_kernel<DKP, MAXT, WT, OT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); attr = true; }
    const int threads = (4 * p.dv + 31) / 32 * 32;
    launch_pdl((delta_step_kernel<DKP, MAXT, WT, OT>), dim3(nseq, p.H), threads, base + (staged ? gates : 0), st, p, staged);
    return (int)cudaGetLastError();
}
template <int DKP, typename WT, typename OT>
static int launch_delta_step(const DeltaParams& p, int nseq, cudaStream_t st) {
    if (p.dv <= 64) return launch_delta_step_t<DKP, 256, WT, OT>(p, nseq, st);
    if (p.dv <= 128) return launch_delta_step_t<DKP, 512, WT, OT>(p, nseq, st);
    if constexpr (DKP <= 64) return launch_delta_step_t<DKP, 1024, WT, OT>(p, nseq, st);
    return -1;
}

template <int DKP, typename OT>
static int launch_delta_rows(const DeltaParams& p, const DeltaScratch& w, int nseq, int total_rows, int short_seqs, int long_seqs, int nchunks, int long_min,
                             float* chunk_ws, cudaStream_t st) {
    launch_pdl((delta_prep_kernel<DKP>), dim3((total_rows + kDeltaPrepRows - 1) / kDeltaPrepRows, p.H), 128, 0, st, p, w, nseq, total_rows);
    if (short_seqs) launch_pdl((delta_recur_kernel<DKP>), dim3(nseq, p.H, (p.dv + 31) / 32), 128, 0, st, p, w, long_seqs ? long_min : (1 << 30));
    if constexpr (DKP <= 128) {
        if (long_seqs) {
            static bool attr = false;
            if (!attr) {
                cudaFuncSetAttribute(delta_chunk_prep_kernel<DKP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ChunkDims<DKP>::kPrepSmem);
                cudaFuncSetAttribute(delta_chunk_scan_kernel<DKP, DeltaTail>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ChunkDims<DKP>::kScanSmem);
                attr = true;
            }
            DeltaChunkArgs ca{w.qn, w.kn, w.ld, w.vo, w.beta, p.state, p.seq_row0, p.seq_nrows, p.seq_slot, nseq, long_min, p.H, p.dv, 1,
                              chunk_ws, chunk_ws + (size_t)nchunks * p.H * kCh * kCh, chunk_ws + (size_t)2 * nchunks * p.H * kCh * kCh};
            launch_pdl((delta_chunk_prep_kernel<DKP>), dim3(nchunks, p.H), 256, ChunkDims<DKP>::kPrepSmem, st, ca);
            launch_pdl((delta_chunk_scan_kernel<DKP, DeltaTail>), dim3(p.H, (p.dv + kCh - 1) / kCh, nseq), 256, ChunkDims<DKP>::kScanSmem, st, ca, DeltaTail{p});
        }
    }
    const long long nrh = (long long)total_rows * p.H;
    launch_pdl((delta_out_kernel<OT>), (unsigned)((nrh + 3) / 4), 128, 0, st, p, w, total_rows);
    return (int)cudaGetLastError();
}

}  // namespace lsb
using namespace lsb;

LSB_API int lsb_gemm_bf16_tc(void* out, const void* x, const void* w, const void* bias, int M, int N, int K, int ldx, int ldw,
                             int ldo, int out_bf16, void* partial, long long partial_cap, void* err, const void* comm, void* stream);
LSB_API int lsb_gemm_f32(void* out, const void* x, const void* w, int M, int N, int K, int ldx, int ldw, int ldo, void* stream);

// padded key width of the state rows and of the row-parallel scratch arrays
LSB_API int lsb_delta_key_pad(int dk) { return dk > 256 || dk < 1 ? -1 : delta_pad(dk); }

// largest value head the one-kernel form takes next to key heads of dk channels
LSB_API int lsb_delta_few_max_dv(int dk) { return delta_step_max_dv(delta_pad(dk)); }

// floats of scratch a step of `rows` rows needs (0: the step kernel takes any step)
LSB_API int lsb_delta_scratch_floats(int rows, int H, int dk, int dv, int rank_a, int rank_g) {
    const long long n = (long long)rows * H * (3 * delta_pad(dk) + dv + 2 + dk + dv) + (long long)rows * (rank_a + rank_g) + 64;
    return n > 0x7fffffffLL ? -1 : (int)n;
}
LSB_API int lsb_delta_chunk_floats(int chunks, int H, int dk) {
    const long long n = (long long)chunks * H * (2 * kCh * kCh + delta_pad(dk));
    return n > 0x7fffffffLL ? -1 : (int)n;
}

// One layer body over the step's rows: proj (the fused input projection) -> out.  rank_a = rank_g = 0: decays per head (dt_bias [H]), full-rank gate.  f32: weights w_a / w_g and `out` are fp32, otherwise bf16;
// w_a2 / w_g2 = [W | W] (bf16 only).  few: the host's choice of the one-kernel form (dv <= lsb_delta_few_max_dv(dk)).  Otherwise scratch is required, with
// `short_seqs` / `long_seqs` = how many sequences have fewer / at least `long_min` rows and `nchunks` = 64-token chunks of the latter
// (long sequences need dk <= 128 and chunk_ws).  gemm_err: error word of the tensor-core products.
LSB_API int lsb_delta_forward(const void* proj, int ldp, int off_q, int off_k, int off_v, int off_b, int off_a, int off_g, int rank_a, int rank_g,
                              const void* w_a, const void* w_g, const void* w_a2, const void* w_g2, const void* conv_q, const void* conv_k,
                              const void* conv_v, const void* a_exp, const void* dt_bias, const void* onorm, void* state, void* conv_state,
                              const void* seq_row0, const void* seq_nrows, const void* seq_slot, void* out, int ldo, int nseq, int total_rows, int H,
                              int G, int dk, int dv, int taps, int decay_mode, float q_scale, float decay_bound, float eps, int f32, int few,
                              void* scratch, int short_seqs, int long_seqs, int nchunks, int long_min, void* chunk_ws, void* gemm_err, void* stream) {
    if (dk < 1 || dk > 256 || dv < 1 || H < 1 || G < 1 || H % G || taps < 1 || rank_a % 8 || rank_g % 8 || total_rows < 1 || nseq < 1) return -1;
    if ((rank_a == 0) != (rank_g == 0)) return -1;
    if (few && dv > delta_step_max_dv(delta_pad(dk))) return -1;
    if (!few && (!scratch || (long_seqs && (dk > 128 || !chunk_ws || long_min < 1)))) return -1;
    cudaStream_t st = (cudaStream_t)stream;
    DeltaParams p;
    p.proj = (const float*)proj; p.ldp = ldp; p.off_q = off_q; p.off_k = off_k; p.off_v = off_v; p.off_b = off_b; p.off_a = off_a; p.off_g = off_g;
    p.rank_a = rank_a; p.rank_g = rank_g; p.w_a = w_a; p.w_g = w_g; p.conv_q = (const float*)conv_q; p.conv_k = (const float*)conv_k;
    p.conv_v = (const float*)conv_v; p.a_exp = (const float*)a_exp; p.dt_bias = (const float*)dt_bias; p.onorm = (const float*)onorm;
    p.state = (float*)state; p.conv_state = (float*)conv_state; p.seq_row0 = (const int*)seq_row0; p.seq_nrows = (const int*)seq_nrows;
    p.seq_slot = (const int*)seq_slot; p.out = out; p.ldo = ldo; p.H = H; p.G = G; p.dk = dk; p.dv = dv; p.taps = taps; p.decay_mode = decay_mode;
    p.q_scale = q_scale; p.decay_bound = decay_bound; p.eps = eps;
    const int DKP = delta_pad(dk);
    if (few) {
#define LSB_STEP(D) return f32 ? launch_delta_step<D, float, float>(p, nseq, st) : launch_delta_step<D, bf16, bf16>(p, nseq, st)
        switch (DKP) { case 32: LSB_STEP(32); case 64: LSB_STEP(64); case 128: LSB_STEP(128); default: LSB_STEP(256); }
#undef LSB_STEP
    }
    const size_t n = (size_t)total_rows * H;
    DeltaScratch w;
    w.qn = (float*)scratch; w.kn = w.qn + n * DKP; w.ld = w.kn + n * DKP;
    w.vo = w.ld + n * DKP; w.beta = w.vo + n * dv; w.kq = w.beta + n; w.rawa = w.kq + n; w.rawg = w.rawa + n * dk;
    float* rest = w.rawg + n * dv;
    int rc;
    if (rank_a == 0 && rank_g == 0) {
        rc = 0;                                                    // nothing low-rank: decays and gates are columns of the projection
    } else if (f32) {
        rc = lsb_gemm_f32(w.rawa, (const float*)proj + off_a, w_a, total_rows, H * dk, rank_a, ldp, rank_a, H * dk, stream);
        if (rc) return rc;
        rc = lsb_gemm_f32(w.rawg, (const float*)proj + off_g, w_g, total_rows, H * dv, rank_g, ldp, rank_g, H * dv, stream);
        if (rc) return rc;
    } else {
        bf16* xs = reinterpret_cast<bf16*>(((uintptr_t)rest + 15) & ~(uintptr_t)15);
        const int ldx = 2 * (rank_a + rank_g);
        launch_pdl((delta_split_kernel), total_rows, 128, 0, st, (const float*)proj, ldp, off_a, rank_a, off_g, rank_g, xs);
        rc = lsb_gemm_bf16_tc(w.rawa, xs, w_a2, nullptr, total_rows, H * dk, 2 * rank_a, ldx, 2 * rank_a, H * dk, 0, nullptr, 0, gemm_err, nullptr, stream);
        if (rc) return rc;
        rc = lsb_gemm_bf16_tc(w.rawg, xs + 2 * rank_a, w_g2, nullptr, total_rows, H * dv, 2 * rank_g, ldx, 2 * rank_g, H * dv, 0, nullptr, 0, gemm_err, nullptr, stream);
        if (rc) return rc;
    }
#define LSB_ROWS(D) return f32 ? launch_delta_rows<D, float>(p, w, nseq, total_rows, short_seqs, long_seqs, nchunks, long_min, (float*)chunk_ws, st) \
                               : launch_delta_rows<D, bf16>(p, w, nseq, total_rows, short_seqs, long_seqs, nchunks, long_min, (float*)chunk_ws, st)
    switch (DKP) { case 32: LSB_ROWS(32); case 64: LSB_ROWS(64); case 128: LSB_ROWS(128); default: LSB_ROWS(256); }
#undef LSB_ROWS
}

LSB_API int lsb_trace_set_delta(void* buf) { return lsb_trace_install(buf); }
