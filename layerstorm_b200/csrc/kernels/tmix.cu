// Time mixing: a linear recurrence with a data-dependent decay per key channel and a bonus for the current token, for any head geometry.
//
//   x_s = h + (h' - h) mu_s,  s in {r, k, v, g, w}        h': the previous token's input of the layer (zeros for the first token)
//   r, k, v = W x;  log w = -exp(W_2 tanh(W_1 x_w) + w_0)                               per head and key channel
//   o = S^T r + (r . (u k)) v,   S <- diag(w) S + k v^T                                 per head
//   out = o / sqrt(mean(o^2) + eps) * w_norm * silu(W_g x_g)
//
// State: fp32 [slots, H, dv, DKP], one row of DKP (dk padded to 32 / 64 / 128 / 256) floats per value channel; the previous token's input: fp32
// [slots, ldx].  A launch that reads another row's predecessor never writes it: tmix_shift reads the kept input, the last kernel of the layer
// replaces it.
//
//   tmix_shift   the five mixed inputs of every row
//   tmix_step    few rows per sequence (and key heads wider than 128): decays, recurrence, gated norm in one kernel
//   longer runs, in chunks of 64 tokens.  The state enters linearly and decays per channel, so only an element-wise scan is sequential:
//   tmix_chunk   per (chunk, head): pair products inside the chunk, its output without the incoming state, its contribution to the state
//   tmix_scan    states in front of every chunk
//   tmix_out     the incoming state's part of the output, gated norm
// With L the cumulative log decay inside a sub-chunk of 16 tokens and T its total: exp(sum of log decays between two tokens) factors into terms whose
// exponents are all <= 0 and sums of few numbers, however strong the decays are.
#include "common.cuh"

namespace lsb {

#include "kda_chunk.cuh"

struct TmixParams {
    const float* proj;                       // [rows, ldp] fp32: r | k | v | g | w (rank of the decay) at the offsets below
    int ldp, off_r, off_k, off_v, off_g, off_w, rank;        // rank padded to a multiple of 8
    const void* w2;                          // [H * dk, rank]
    const float* w0; const float* u;         // [H * dk]
    const float* onorm;                      // [H * dv]
    float* state; float* prev;
    const void* x; int ldx;                  // the layer's input rows (activation type)
    const int* seq_row0; const int* seq_nrows; const int* seq_slot;
    void* out; int ldo;
    int H, dk, dv;
    float eps;
};

struct TmixScratch {
    float* rawd;      // [rows, H * dk]        W_2 tanh(..)
    float* qp;        // [rows, H, DK]         r times the decay since the chunk's start
    float* o;         // [rows, H, dv]
    float* kv;        // [chunks, H, dv, DK]   a chunk's contribution to the state, then the state in front of it
    float* gc;        // [chunks, H, DK]       decay over the chunk
};

template <typename T> __device__ __forceinline__ float act_in(T v);
template <> __device__ __forceinline__ float act_in<bf16>(bf16 v) { return __bfloat162float(v); }
template <> __device__ __forceinline__ float act_in<float>(float v) { return v; }
template <typename T> __device__ __forceinline__ T act_out(float v);
template <> __device__ __forceinline__ bf16 act_out<bf16>(float v) { return __float2bfloat16(v); }
template <> __device__ __forceinline__ float act_out<float>(float v) { return v; }
__device__ __forceinline__ float tmix_silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float tmix_quad_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    return v + __shfl_xor_sync(0xffffffffu, v, 2);
}
// logarithm of a decay factor; below exp(-100) a factor is 0 in fp32, and sums of 64 of them stay exact enough
__device__ __forceinline__ float tmix_log_decay(float x) { return fmaxf(-expf(x), -100.f); }

// keeps the last row of a sequence as its next token's predecessor (one block)
template <typename T>
__device__ __forceinline__ void tmix_keep(const TmixParams& p, int seq, int slot) {
    const T* x = reinterpret_cast<const T*>(p.x) + (size_t)(p.seq_row0[seq] + p.seq_nrows[seq] - 1) * p.ldx;
    for (int c = threadIdx.x; c < p.ldx; c += blockDim.x) p.prev[(size_t)slot * p.ldx + c] = act_in<T>(x[c]);
}

// ------------------------------------------------------------------------------------------------ token shift
// xs[s][row] = x[row] + (x[row - 1] - x[row]) * mu[s], s < 5; the first row of a sequence takes its predecessor from `prev`.
template <typename T>
__global__ void __launch_bounds__(256) tmix_shift_kernel(const T* __restrict__ x, int ldx, const float* __restrict__ prev, const float* __restrict__ mu,
                                                         T* __restrict__ xs, long long stride, const int* __restrict__ seq_row0,
                                                         const int* __restrict__ seq_nrows, const int* __restrict__ seq_slot, int nseq) {
    __shared__ int s_slot;
    const int row = blockIdx.x;
    const int c = (blockIdx.y * 256 + threadIdx.x) * 4;
    float4 m[5];
    if (c < ldx) {
#pragma unroll
        for (int s = 0; s < 5; ++s) m[s] = *reinterpret_cast<const float4*>(mu + (size_t)s * ldx + c);
    }
    if (threadIdx.x == 0) s_slot = -1;
    pdl_wait();
    pdl_launch_dependents();
    __syncthreads();
    for (int s = threadIdx.x; s < nseq; s += 256)
        if (seq_row0[s] == row && seq_nrows[s] > 0) s_slot = seq_slot[s];
    __syncthreads();
    if (c >= ldx) return;
    float h[4], d[4];
    const T* xr = x + (size_t)row * ldx + c;
#pragma unroll
    for (int e = 0; e < 4; ++e) h[e] = act_in<T>(xr[e]);
    if (s_slot >= 0) {
        const float4 q = *reinterpret_cast<const float4*>(prev + (size_t)s_slot * ldx + c);
        d[0] = q.x; d[1] = q.y; d[2] = q.z; d[3] = q.w;
    } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) d[e] = row > 0 ? act_in<T>(xr[e - ldx]) : 0.f;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) d[e] -= h[e];
#pragma unroll
    for (int s = 0; s < 5; ++s) {
        T* o = xs + s * stride + (size_t)row * ldx + c;
        const float mm[4] = {m[s].x, m[s].y, m[s].z, m[s].w};
        if constexpr (sizeof(T) == 2) {
            bf162 v[2];
            v[0] = __floats2bfloat162_rn(fmaf(d[0], mm[0], h[0]), fmaf(d[1], mm[1], h[1]));
            v[1] = __floats2bfloat162_rn(fmaf(d[2], mm[2], h[2]), fmaf(d[3], mm[3], h[3]));
            *reinterpret_cast<uint2*>(o) = *reinterpret_cast<const uint2*>(v);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) o[e] = fmaf(d[e], mm[e], h[e]);
        }
    }
}

// ------------------------------------------------------------------------------------------------ few rows
constexpr int kTmixGroup = 8;         // rows whose decays and keys are prepared together

// dot of a row of the low-rank decay matrix with an fp32 vector over the four lanes of a quad
template <typename T> __device__ __forceinline__ float tmix_dot(const T* row, const float* x, int rank, int ks) {
    float a = 0.f;
    if constexpr (sizeof(T) == 2) {
        for (int j = ks * 8; j < rank; j += 32) {
            float f[8];
            unpack_bf16x8(*reinterpret_cast<const uint4*>(row + j), f);
#pragma unroll
            for (int e = 0; e < 8; ++e) a = fmaf(f[e], x[j + e], a);
        }
    } else {
        for (int j = ks * 4; j < rank; j += 16) {
            const float4 f = *reinterpret_cast<const float4*>(row + j);
            a = fmaf(f.x, x[j], a); a = fmaf(f.y, x[j + 1], a); a = fmaf(f.z, x[j + 2], a); a = fmaf(f.w, x[j + 3], a);
        }
    }
    return tmix_quad_sum(a);
}

// One block per (sequence, head), four threads per value channel; value heads wider than the block go in tiles.
template <int DKP, int MAXT, typename T>
__global__ void __launch_bounds__(MAXT, 1) tmix_step_kernel(TmixParams p) {
    constexpr int NJ = DKP / 16;
    extern __shared__ __align__(16) float tsm[];
    const int nt = blockDim.x, t = threadIdx.x, lane = t & 31, warp = t >> 5, ks = t & 3, VT = nt >> 2;
    const int seq = blockIdx.x, h = blockIdx.y;
    float* s_r = tsm;                                              // [8][DKP]
    float* s_k = s_r + kTmixGroup * DKP;
    float* s_w = s_k + kTmixGroup * DKP;                           // decay factors
    float* s_a = s_w + kTmixGroup * DKP;                           // [8][rank]
    float* s_o = s_a + kTmixGroup * p.rank;                        // [8][dv]
    float* s_b = s_o + kTmixGroup * p.dv;                          // [8]   r . (u k)
    const int row0 = p.seq_row0[seq], nrows = p.seq_nrows[seq], slot = p.seq_slot[seq];
    const bool live = nrows > 0 && slot >= 0, one = p.dv <= VT;
    const T* w2 = reinterpret_cast<const T*>(p.w2) + (size_t)h * p.dk * p.rank;
    for (int i = t * (128 / (int)sizeof(T)); i < p.dk * p.rank; i += nt * (128 / (int)sizeof(T))) asm volatile("prefetch.global.L2 [%0];" ::"l"(w2 + i));
    float* sp = p.state + ((size_t)(live ? slot : 0) * p.H + h) * p.dv * DKP + ks * 4;
    float4 S[NJ];
    auto load = [&](int v) {
#pragma unroll
        for (int j = 0; j < NJ; ++j) S[j] = v < p.dv ? *reinterpret_cast<const float4*>(sp + (size_t)v * DKP + j * 16) : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    auto store = [&](int v) {
        if (v < p.dv) {
#pragma unroll
            for (int j = 0; j < NJ; ++j) *reinterpret_cast<float4*>(sp + (size_t)v * DKP + j * 16) = S[j];
        }
    };
    if (live && one) load(t >> 2);
    pdl_wait();
    pdl_launch_dependents();
    if (!live) return;
    for (int g0 = 0; g0 < nrows; g0 += kTmixGroup) {
        const int m = min(kTmixGroup, nrows - g0);
        const float* pr = p.proj + (size_t)(row0 + g0) * p.ldp;
        for (int i = t; i < m * DKP; i += nt) {
            const int r = i / DKP, c = i % DKP;
            s_r[i] = c < p.dk ? pr[(size_t)r * p.ldp + p.off_r + h * p.dk + c] : 0.f;
            s_k[i] = c < p.dk ? pr[(size_t)r * p.ldp + p.off_k + h * p.dk + c] : 0.f;
            if (c >= p.dk) s_w[i] = 0.f;
        }
        for (int i = t; i < m * p.rank; i += nt) s_a[i] = tanhf(pr[(size_t)(i / p.rank) * p.ldp + p.off_w + i % p.rank]);
        __syncthreads();
        for (int c0 = 0; c0 < p.dk; c0 += VT) {
            const int c = c0 + (t >> 2);
            for (int r = 0; r < m; ++r) {
                const float x = tmix_dot<T>(w2 + (size_t)min(c, p.dk - 1) * p.rank, s_a + r * p.rank, p.rank, ks);
                if (ks == 0 && c < p.dk) s_w[r * DKP + c] = expf(tmix_log_decay(x + p.w0[(size_t)h * p.dk + c]));
            }
        }
        for (int r = warp; r < m; r += nt >> 5) {
            float a = 0.f;
            for (int c = lane; c < p.dk; c += 32) a = fmaf(s_r[r * DKP + c] * p.u[(size_t)h * p.dk + c], s_k[r * DKP + c], a);
            a = warp_sum(a);
            if (lane == 0) s_b[r] = a;
        }
        __syncthreads();
        for (int v0 = 0; v0 < p.dv; v0 += VT) {
            const int v = v0 + (t >> 2);
            if (!one) load(v);
            for (int r = 0; r < m; ++r) {
                const float vv = v < p.dv ? pr[(size_t)r * p.ldp + p.off_v + h * p.dv + v] : 0.f;
                const float4* r4 = reinterpret_cast<const float4*>(s_r + r * DKP) + ks;
                const float4* k4 = reinterpret_cast<const float4*>(s_k + r * DKP) + ks;
                const float4* w4 = reinterpret_cast<const float4*>(s_w + r * DKP) + ks;
                float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const float4 q = r4[j * 4], k = k4[j * 4], w = w4[j * 4];
                    a.x = fmaf(S[j].x, q.x, a.x); a.y = fmaf(S[j].y, q.y, a.y); a.z = fmaf(S[j].z, q.z, a.z); a.w = fmaf(S[j].w, q.w, a.w);
                    S[j].x = fmaf(S[j].x, w.x, k.x * vv); S[j].y = fmaf(S[j].y, w.y, k.y * vv);
                    S[j].z = fmaf(S[j].z, w.z, k.z * vv); S[j].w = fmaf(S[j].w, w.w, k.w * vv);
                }
                const float o = tmix_quad_sum((a.x + a.y) + (a.z + a.w));
                if (ks == 0 && v < p.dv) s_o[r * p.dv + v] = fmaf(vv, s_b[r], o);
            }
            if (!one) store(v);
        }
        __syncthreads();
        for (int r = warp; r < m; r += nt >> 5) {
            float q = 0.f;
            for (int c = lane; c < p.dv; c += 32) q = fmaf(s_o[r * p.dv + c], s_o[r * p.dv + c], q);
            const float rs = 1.f / sqrtf(warp_sum(q) / (float)p.dv + p.eps);
            for (int c = lane; c < p.dv; c += 32)
                reinterpret_cast<T*>(p.out)[(size_t)(row0 + g0 + r) * p.ldo + (size_t)h * p.dv + c] =
                    act_out<T>(s_o[r * p.dv + c] * rs * p.onorm[(size_t)h * p.dv + c] * tmix_silu(pr[(size_t)r * p.ldp + p.off_g + h * p.dv + c]));
        }
        __syncthreads();
    }
    if (one) store(t >> 2);
    if (h == 0) tmix_keep<T>(p, seq, slot);
}

// ------------------------------------------------------------------------------------------------ many rows
// tanh of the low-rank activations: fp32 rows, or bf16 (hi | lo) pairs that with the duplicated weights [W | W] give the product to ~2^-16
template <typename T>
__global__ void __launch_bounds__(128) tmix_tanh_kernel(const float* __restrict__ proj, int ldp, int off, int rank, T* __restrict__ out) {
    pdl_wait();
    pdl_launch_dependents();
    const int row = blockIdx.x;
    for (int j = threadIdx.x; j < rank; j += 128) {
        const float v = tanhf(proj[(size_t)row * ldp + off + j]);
        if constexpr (sizeof(T) == 2) {
            const bf16 hi = __float2bfloat16(v);
            out[(size_t)row * 2 * rank + j] = hi;
            out[(size_t)row * 2 * rank + rank + j] = __float2bfloat16(v - __bfloat162float(hi));
        } else {
            out[(size_t)row * rank + j] = v;
        }
    }
}

// chunk number (over the step's sequences in order) -> rows [row0 + c0, + cc) of sequence seq; cc 0: no such chunk
__device__ __forceinline__ void tmix_find(const TmixParams& p, int nseq, int chunk, int& seq, int& row0, int& c0, int& cc) {
    seq = row0 = c0 = cc = 0;
    for (int s = 0, base = 0; s < nseq; ++s) {
        const int n = p.seq_nrows[s], nc = (n + kCh - 1) / kCh;
        if (chunk < base + nc) { seq = s; row0 = p.seq_row0[s]; c0 = (chunk - base) * kCh; cc = min(kCh, n - c0); return; }
        base += nc;
    }
}

template <int DK> struct TmixDims {
    static constexpr int kLdK = DK + 4, kLdR = DK + 1;
    static constexpr size_t kChunkSmem = (size_t)(3 * kCh * kLdK + 2 * kCh * kLdC + (kSub + kCh - kSub) * kLdR) * sizeof(float);
    static constexpr size_t kOutSmem = (size_t)(2 * kCh * kLdK) * sizeof(float);
};

template <int kD>
__global__ void __launch_bounds__(256) tmix_chunk_kernel(TmixParams p, TmixScratch w, int nseq) {
    constexpr int kLdK = TmixDims<kD>::kLdK, kLdR = TmixDims<kD>::kLdR, NK = kD / 16;
    extern __shared__ __align__(16) float csm[];
    float* sR = csm;                          // [t][c] r
    float* sK = sR + kCh * kLdK;              // [t][c] k
    float* sL = sK + kCh * kLdK;              // [t][c] log decay, then its sum over the sub-chunk up to and including t
    float* sA = sL + kCh * kLdK;              // [t][s] pair products
    float* sV = sA + kCh * kLdC;              // [v][t] values of a tile
    float* sX = sV + kCh * kLdC;              // [16][kLdR] rescaled r rows of a sub-chunk;  first, with sY: [64][kLdR] decay factors
    float* sY = sX + kSub * kLdR;             // [48][kLdR] rescaled earlier k rows
    const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, tx = tid & 15, ty = tid >> 4;
    pdl_wait();
    pdl_launch_dependents();
    int seq, row0, c0, cc;
    tmix_find(p, nseq, chunk, seq, row0, c0, cc);
    if (cc <= 0 || p.seq_slot[seq] < 0) return;
    const int r0 = row0 + c0, dk = p.dk;
#pragma unroll 8
    for (int idx = tid; idx < kCh * kD; idx += 256) {
        const int t = idx / kD, c = idx % kD;
        float r = 0.f, k = 0.f, l = 0.f;
        if (t < cc && c < dk) {
            const float* pr = p.proj + (size_t)(r0 + t) * p.ldp + h * dk + c;
            r = pr[p.off_r];
            k = pr[p.off_k];
            l = tmix_log_decay(w.rawd[(size_t)(r0 + t) * p.H * dk + h * dk + c] + p.w0[(size_t)h * dk + c]);
        }
        sR[t * kLdK + c] = r; sK[t * kLdK + c] = k; sL[t * kLdK + c] = l;
        sX[t * kLdR + c] = expf(l);
    }
    for (int idx = tid; idx < kCh * kLdC; idx += 256) sA[idx] = 0.f;
    __syncthreads();
    for (int idx = tid; idx < (kCh / kSub) * kD; idx += 256) {
        float* l = sL + (idx / kD) * kSub * kLdK + idx % kD;
        float acc = 0.f;
        for (int t = 0; t < kSub; ++t) { acc += l[t * kLdK]; l[t * kLdK] = acc; }
    }
    __syncthreads();
    auto total = [&](int sub, int c) { return sL[(sub * kSub + kSub - 1) * kLdK + c]; };
    // pair products inside the sub-chunks: a warp takes a row t and walks back over its predecessors, the factors between them multiplied up in
    // registers; the 16 sums over the lanes' channels are folded together, lane 2 d ends up with the one of distance d
    for (int t = warp; t < cc; t += 8) {
        const int dt = t % kSub;
        float P[kD / 32], a[kSub];
#pragma unroll
        for (int i = 0; i < kD / 32; ++i) P[i] = sR[t * kLdK + lane + 32 * i];
#pragma unroll
        for (int d = 0; d < kSub; ++d) {
            a[d] = 0.f;
            if (d > dt) continue;                              // warp-uniform
#pragma unroll
            for (int i = 0; i < kD / 32; ++i) {
                const int c = lane + 32 * i;
                const float k = sK[(t - d) * kLdK + c];
                if (d == 0) {
                    a[d] = fmaf(P[i] * (c < dk ? p.u[(size_t)h * dk + c] : 0.f), k, a[d]);
                } else {
                    a[d] = fmaf(P[i], k, a[d]);
                    P[i] *= sX[(t - d) * kLdR + c];
                }
            }
        }
#pragma unroll
        for (int o = 16, n = kSub / 2; n >= 1; o >>= 1, n >>= 1) {
#pragma unroll
            for (int j = 0; j < kSub / 2; ++j) {
                if (j >= n) break;
                const float give = lane & o ? a[j] : a[j + n], keep = lane & o ? a[j + n] : a[j];
                a[j] = keep + __shfl_xor_sync(0xffffffffu, give, o);
            }
        }
        a[0] += __shfl_xor_sync(0xffffffffu, a[0], 1);
        const int d = lane >> 1;
        if ((lane & 1) == 0 && d <= dt) sA[t * kLdC + t - d] = a[0];
    }
    __syncthreads();                                           // sX and sY are refilled next
    // against earlier sub-chunks: a product of two rescaled tiles
    for (int I = 1; I < kCh / kSub; ++I) {
        const int t0 = I * kSub;
        if (t0 >= cc) break;                                   // block-uniform
        for (int idx = tid; idx < kSub * kD; idx += 256) {
            const int tt = idx / kD, c = idx % kD;
            sX[tt * kLdR + c] = sR[(t0 + tt) * kLdK + c] * (tt ? expf(sL[(t0 + tt - 1) * kLdK + c]) : 1.f);
        }
        for (int idx = tid; idx < t0 * kD; idx += 256) {
            const int s = idx / kD, c = idx % kD, J = s / kSub;
            float e = total(J, c) - sL[s * kLdK + c];
            for (int K = J + 1; K < I; ++K) e += total(K, c);
            sY[s * kLdR + c] = sK[s * kLdK + c] * expf(fminf(e, 0.f));
        }
        __syncthreads();
        for (int o = tid; o < kSub * t0; o += 256) {
            const int tt = o / t0, s = o - tt * t0;
            const float* xr = sX + tt * kLdR;
            const float* yr = sY + s * kLdR;
            float a0 = 0.f, a1 = 0.f;
#pragma unroll 8
            for (int c = 0; c < kD; c += 2) { a0 = fmaf(xr[c], yr[c], a0); a1 = fmaf(xr[c + 1], yr[c + 1], a1); }
            if (t0 + tt < cc) sA[(t0 + tt) * kLdC + s] = a0 + a1;
        }
        __syncthreads();                                       // the tiles are rebuilt for the next sub-chunk
    }
    __syncthreads();
    // r and k times the decays from the chunk's start and to its end; the chunk's whole decay
#pragma unroll 4
    for (int idx = tid; idx < kCh * kD; idx += 256) {
        const int t = idx / kD, c = idx % kD, J = t / kSub;
        float before = t % kSub ? sL[(t - 1) * kLdK + c] : 0.f, after = total(J, c) - sL[t * kLdK + c];
        for (int K = 0; K < J; ++K) before += total(K, c);
        for (int K = J + 1; K < kCh / kSub; ++K) after += total(K, c);
        if (t < cc) w.qp[((size_t)(r0 + t) * p.H + h) * kD + c] = sR[t * kLdK + c] * expf(before);
        sK[t * kLdK + c] *= expf(fminf(after, 0.f));
        if (t == 0) w.gc[((size_t)chunk * p.H + h) * kD + c] = expf(total(0, c) + total(1, c) + total(2, c) + total(3, c));
    }
    __syncthreads();
    for (int v0 = 0; v0 < p.dv; v0 += kCh) {
#pragma unroll 8
        for (int idx = tid; idx < kCh * kCh; idx += 256) {
            const int t = idx / kCh, v = idx % kCh;
            sV[v * kLdC + t] = t < cc && v0 + v < p.dv ? p.proj[(size_t)(r0 + t) * p.ldp + p.off_v + h * p.dv + v0 + v] : 0.f;
        }
        __syncthreads();
        float acc[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
        kda_mm_nt<kCh>(sA, kLdC, sV, kLdC, acc, tx, ty);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int t = ty + 16 * i, v = v0 + tx + 16 * j;
                if (t < cc && v < p.dv) w.o[((size_t)(r0 + t) * p.H + h) * p.dv + v] = acc[i][j];
            }
        float a2[4][NK];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < NK; ++j) a2[i][j] = 0.f;
#pragma unroll 2
        for (int t = 0; t < kCh; ++t) {
            float u[4], km[NK];
#pragma unroll
            for (int i = 0; i < 4; ++i) u[i] = sV[(ty + 16 * i) * kLdC + t];
#pragma unroll
            for (int j = 0; j < NK; ++j) km[j] = sK[t * kLdK + tx + 16 * j];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < NK; ++j) a2[i][j] = fmaf(u[i], km[j], a2[i][j]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int v = v0 + ty + 16 * i;
            if (v < p.dv) {
#pragma unroll
                for (int j = 0; j < NK; ++j) w.kv[(((size_t)chunk * p.H + h) * p.dv + v) * kD + tx + 16 * j] = a2[i][j];
            }
        }
        __syncthreads();
    }
}

// states in front of every chunk (in place of the chunks' contributions) and behind the last: one thread per four key channels of a value channel
__global__ void __launch_bounds__(256) tmix_scan_kernel(TmixParams p, TmixScratch w, int kD) {
    const int seq = blockIdx.z, h = blockIdx.y, i = (blockIdx.x * 256 + threadIdx.x) * 4;
    pdl_wait();
    pdl_launch_dependents();
    const int slot = p.seq_slot[seq], nc = (p.seq_nrows[seq] + kCh - 1) / kCh, n = p.dv * kD;
    if (i >= n || slot < 0 || nc <= 0) return;
    int base = 0;
    for (int s = 0; s < seq; ++s) base += (p.seq_nrows[s] + kCh - 1) / kCh;
    float4* st = reinterpret_cast<float4*>(p.state + ((size_t)slot * p.H + h) * n + i);
    float4 S = *st;
    const size_t skv = (size_t)p.H * n, sg = (size_t)p.H * kD;
    float* kv = w.kv + ((size_t)base * p.H + h) * n + i;
    const float* gc = w.gc + ((size_t)base * p.H + h) * kD + i % kD;
    for (int c0 = 0; c0 < nc; c0 += 8) {
        float4 a[8], g[8];
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (c0 + j < nc) { a[j] = *reinterpret_cast<const float4*>(kv + (c0 + j) * skv); g[j] = *reinterpret_cast<const float4*>(gc + (c0 + j) * sg); }
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (c0 + j < nc) {
                *reinterpret_cast<float4*>(kv + (c0 + j) * skv) = S;
                S.x = fmaf(S.x, g[j].x, a[j].x); S.y = fmaf(S.y, g[j].y, a[j].y); S.z = fmaf(S.z, g[j].z, a[j].z); S.w = fmaf(S.w, g[j].w, a[j].w);
            }
    }
    *st = S;
}

// ONE: value heads of up to 64 channels, whose outputs stay in registers up to the norm
template <int kD, bool ONE, typename T>
__global__ void __launch_bounds__(256) tmix_out_kernel(TmixParams p, TmixScratch w, int nseq) {
    constexpr int kLdK = TmixDims<kD>::kLdK;
    extern __shared__ __align__(16) float csm[];
    float* sQ = csm;                          // [t][c]
    float* sS = sQ + kCh * kLdK;              // [v][c]
    const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, tx = tid & 15, ty = tid >> 4;
    pdl_wait();
    pdl_launch_dependents();
    int seq, row0, c0, cc;
    tmix_find(p, nseq, chunk, seq, row0, c0, cc);
    if (cc <= 0 || p.seq_slot[seq] < 0) return;
    const int r0 = row0 + c0;
#pragma unroll
    for (int idx = tid; idx < kCh * (kD / 4); idx += 256) {
        const int t = idx / (kD / 4), c4 = idx % (kD / 4) * 4;
        *reinterpret_cast<float4*>(sQ + t * kLdK + c4) =
            t < cc ? *reinterpret_cast<const float4*>(w.qp + ((size_t)(r0 + t) * p.H + h) * kD + c4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float acc[4][4], g[4][4];
    for (int v0 = 0; v0 < p.dv; v0 += kCh) {
#pragma unroll
        for (int idx = tid; idx < kCh * (kD / 4); idx += 256) {
            const int v = idx / (kD / 4), c4 = idx % (kD / 4) * 4;
            *reinterpret_cast<float4*>(sS + v * kLdK + c4) =
                v0 + v < p.dv ? *reinterpret_cast<const float4*>(w.kv + (((size_t)chunk * p.H + h) * p.dv + v0 + v) * kD + c4) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int t = ty + 16 * i, v = v0 + tx + 16 * j;
                const bool in = t < cc && v < p.dv;
                acc[i][j] = in ? w.o[((size_t)(r0 + t) * p.H + h) * p.dv + v] : 0.f;
                if (ONE) g[i][j] = in ? p.proj[(size_t)(r0 + t) * p.ldp + p.off_g + h * p.dv + v] : 0.f;
            }
        __syncthreads();
        kda_mm_nt<kD>(sQ, kLdK, sS, kLdK, acc, tx, ty);
        if (ONE) break;
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int t = ty + 16 * i, v = v0 + tx + 16 * j;
                if (t < cc && v < p.dv) w.o[((size_t)(r0 + t) * p.H + h) * p.dv + v] = acc[i][j];
            }
        __syncthreads();
    }
    if constexpr (ONE) {
        float on[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) on[j] = tx + 16 * j < p.dv ? p.onorm[(size_t)h * p.dv + tx + 16 * j] : 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int t = ty + 16 * i;
            float q = 0.f;
#pragma unroll
            for (int j = 0; j < 4; ++j) q = fmaf(acc[i][j], acc[i][j], q);          // columns past dv hold zeros
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
            const float rs = 1.f / sqrtf(q / (float)p.dv + p.eps);
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (t < cc && tx + 16 * j < p.dv)
                    reinterpret_cast<T*>(p.out)[(size_t)(r0 + t) * p.ldo + (size_t)h * p.dv + tx + 16 * j] = act_out<T>(acc[i][j] * rs * on[j] * tmix_silu(g[i][j]));
        }
    } else {
        for (int t = warp; t < cc; t += 8) {
            const float* o = w.o + ((size_t)(r0 + t) * p.H + h) * p.dv;
            const float* gr = p.proj + (size_t)(r0 + t) * p.ldp + p.off_g + h * p.dv;
            float q = 0.f;
            for (int c = lane; c < p.dv; c += 32) q = fmaf(o[c], o[c], q);
            const float rs = 1.f / sqrtf(warp_sum(q) / (float)p.dv + p.eps);
            for (int c = lane; c < p.dv; c += 32)
                reinterpret_cast<T*>(p.out)[(size_t)(r0 + t) * p.ldo + (size_t)h * p.dv + c] = act_out<T>(o[c] * rs * p.onorm[(size_t)h * p.dv + c] * tmix_silu(gr[c]));
        }
    }
    if (h == 0 && c0 + cc == p.seq_nrows[seq]) tmix_keep<T>(p, seq, p.seq_slot[seq]);
}

static int tmix_pad(int dk) { return dk <= 32 ? 32 : (dk <= 64 ? 64 : (dk <= 128 ? 128 : 256)); }

template <int DKP, int MAXT, typename T>
static int launch_tmix_step(const TmixParams& p, int nseq, cudaStream_t st) {
    const int threads = 4 * p.dv >= MAXT ? MAXT : (4 * p.dv + 31) / 32 * 32;
    const size_t smem = (size_t)(kTmixGroup * (3 * DKP + p.rank + p.dv + 1)) * 4;
    if (smem > 200 * 1024) return -1;
    static bool attr = false;
    if (!attr) { cudaFuncSetAttribute(tmix_step_kernel<DKP, MAXT, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); attr = true; }
    launch_pdl((tmix_step_kernel<DKP, MAXT, T>), dim3(nseq, p.H), threads, smem, st, p);
    return (int)cudaGetLastError();
}

template <int DKP, typename T>
static int launch_tmix_chunks(const TmixParams& p, const TmixScratch& w, int nseq, int nchunks, cudaStream_t st) {
    static bool attr = false;
    if (!attr) {
        cudaFuncSetAttribute(tmix_chunk_kernel<DKP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TmixDims<DKP>::kChunkSmem);
        cudaFuncSetAttribute(tmix_out_kernel<DKP, true, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TmixDims<DKP>::kOutSmem);
        cudaFuncSetAttribute(tmix_out_kernel<DKP, false, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TmixDims<DKP>::kOutSmem);
        attr = true;
    }
    launch_pdl((tmix_chunk_kernel<DKP>), dim3(nchunks, p.H), 256, TmixDims<DKP>::kChunkSmem, st, p, w, nseq);
    launch_pdl((tmix_scan_kernel), dim3((p.dv * DKP / 4 + 255) / 256, p.H, nseq), 256, 0, st, p, w, DKP);
    if (p.dv <= kCh) launch_pdl((tmix_out_kernel<DKP, true, T>), dim3(nchunks, p.H), 256, TmixDims<DKP>::kOutSmem, st, p, w, nseq);
    else launch_pdl((tmix_out_kernel<DKP, false, T>), dim3(nchunks, p.H), 256, TmixDims<DKP>::kOutSmem, st, p, w, nseq);
    return (int)cudaGetLastError();
}

}  // namespace lsb
using namespace lsb;

LSB_API int lsb_gemm_bf16_tc(void* out, const void* x, const void* w, const void* bias, int M, int N, int K, int ldx, int ldw,
                             int ldo, int out_bf16, void* partial, long long partial_cap, void* err, const void* comm, void* stream);
LSB_API int lsb_gemm_f32(void* out, const void* x, const void* w, int M, int N, int K, int ldx, int ldw, int ldo, void* stream);

// padded key width of the state rows
LSB_API int lsb_tmix_key_pad(int dk) { return dk > 256 || dk < 1 ? -1 : tmix_pad(dk); }

// floats of scratch of the chunked form (-1: more than 2^31)
LSB_API int lsb_tmix_scratch_floats(int rows, int chunks, int H, int dk, int dv, int rank) {
    const long long DK = tmix_pad(dk);
    const long long n = (long long)rows * H * (DK + dv + dk) + (long long)rows * rank + (long long)chunks * H * (dv + 1) * DK + 64;
    return n > 0x7fffffffLL ? -1 : (int)n;
}

// The five mixed inputs of every row: xs [5][stride] <- x [rows, ldx]; mu fp32 [5, ldx]; prev fp32 [slots, ldx].  ldx a multiple of 4.
LSB_API int lsb_tmix_shift(const void* x, int ldx, const void* prev, const void* mu, void* xs, long long stride, const void* seq_row0, const void* seq_nrows,
                           const void* seq_slot, int nseq, int rows, int f32, void* stream) {
    if (rows < 1 || nseq < 1 || ldx % 4 || stride % 8) return -1;
    const dim3 grid(rows, (ldx / 4 + 255) / 256);
    cudaStream_t st = (cudaStream_t)stream;
    if (f32) launch_pdl((tmix_shift_kernel<float>), grid, 256, 0, st, (const float*)x, ldx, (const float*)prev, (const float*)mu, (float*)xs, stride, (const int*)seq_row0,
                        (const int*)seq_nrows, (const int*)seq_slot, nseq);
    else launch_pdl((tmix_shift_kernel<bf16>), grid, 256, 0, st, (const bf16*)x, ldx, (const float*)prev, (const float*)mu, (bf16*)xs, stride, (const int*)seq_row0,
                    (const int*)seq_nrows, (const int*)seq_slot, nseq);
    LSB_CHECK_LAUNCH();
}

// Recurrence, gated norm and state of the step's rows: proj -> out.  f32: w2 and out are fp32, otherwise bf16; w22 = [W_2 | W_2] (bf16, chunked form).
// few: the host's choice of the one-kernel form (any number of rows, token by token).  Otherwise dk <= 128, scratch of lsb_tmix_scratch_floats and the
// number of 64-token chunks over all sequences.  x: the layer's input rows, whose last ones are kept in prev.
LSB_API int lsb_tmix_forward(const void* proj, int ldp, int off_r, int off_k, int off_v, int off_g, int off_w, int rank, const void* w2, const void* w22,
                             const void* w0, const void* u, const void* onorm, void* state, void* prev, const void* x, int ldx, const void* seq_row0,
                             const void* seq_nrows, const void* seq_slot, void* out, int ldo, int nseq, int total_rows, int H, int dk, int dv, float eps, int f32,
                             int few, void* scratch, int nchunks, void* gemm_err, void* stream) {
    if (dk < 1 || dk > 256 || dv < 1 || H < 1 || rank < 8 || rank % 8 || total_rows < 1 || nseq < 1) return -1;
    if (!few && (dk > 128 || !scratch || nchunks < 1 || (!f32 && !w22))) return -1;
    cudaStream_t st = (cudaStream_t)stream;
    TmixParams p;
    p.proj = (const float*)proj; p.ldp = ldp; p.off_r = off_r; p.off_k = off_k; p.off_v = off_v; p.off_g = off_g; p.off_w = off_w; p.rank = rank;
    p.w2 = w2; p.w0 = (const float*)w0; p.u = (const float*)u; p.onorm = (const float*)onorm; p.state = (float*)state; p.prev = (float*)prev;
    p.x = x; p.ldx = ldx; p.seq_row0 = (const int*)seq_row0; p.seq_nrows = (const int*)seq_nrows; p.seq_slot = (const int*)seq_slot;
    p.out = out; p.ldo = ldo; p.H = H; p.dk = dk; p.dv = dv; p.eps = eps;
    const int DKP = tmix_pad(dk);
    if (few) {
#define LSB_TS(D, M) return f32 ? launch_tmix_step<D, M, float>(p, nseq, st) : launch_tmix_step<D, M, bf16>(p, nseq, st)
        switch (DKP) { case 32: LSB_TS(32, 512); case 64: LSB_TS(64, 512); case 128: LSB_TS(128, 512); default: LSB_TS(256, 256); }
#undef LSB_TS
    }
    const size_t n = (size_t)total_rows * H;
    TmixScratch w;
    w.qp = (float*)scratch; w.kv = w.qp + n * DKP; w.gc = w.kv + (size_t)nchunks * H * dv * DKP; w.o = w.gc + (size_t)nchunks * H * DKP; w.rawd = w.o + n * dv;
    void* th = reinterpret_cast<void*>(((uintptr_t)(w.rawd + n * dk) + 15) & ~(uintptr_t)15);
    int rc;
    if (f32) {
        launch_pdl((tmix_tanh_kernel<float>), total_rows, 128, 0, st, (const float*)proj, ldp, off_w, rank, (float*)th);
        rc = lsb_gemm_f32(w.rawd, th, w2, total_rows, H * dk, rank, rank, rank, H * dk, stream);
    } else {
        launch_pdl((tmix_tanh_kernel<bf16>), total_rows, 128, 0, st, (const float*)proj, ldp, off_w, rank, (bf16*)th);
        rc = lsb_gemm_bf16_tc(w.rawd, th, w22, nullptr, total_rows, H * dk, 2 * rank, 2 * rank, 2 * rank, H * dk, 0, nullptr, 0, gemm_err, nullptr, stream);
    }
    if (rc) return rc;
#define LSB_TC(D) return f32 ? launch_tmix_chunks<D, float>(p, w, nseq, nchunks, st) : launch_tmix_chunks<D, bf16>(p, w, nseq, nchunks, st)
    switch (DKP) { case 32: LSB_TC(32); case 64: LSB_TC(64); default: LSB_TC(128); }
#undef LSB_TC
}

LSB_API int lsb_trace_set_tmix(void* buf) { return lsb_trace_install(buf); }
